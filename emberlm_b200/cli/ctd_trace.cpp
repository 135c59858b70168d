// ctd_trace: replays given token ids through a model step by step and writes logits; it samples nothing.
//
//   ctd_trace --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N]
//
// Steps come on standard input, one JSON object a line:
//   {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
// Every entry appends its tokens to request `id` (a new id starts an empty sequence) with
// ctdk_decode_extend, the call generation uses for prompts; `want` are places among these tokens. When
// something is wanted, OUT/<step>.f32 receives the logits [wanted, vocab] (little-endian fp32) in the
// order of the entries. Then "done <step>" goes to standard output. Requests in `end` are finished:
// their sequence is reset and used again. At the end of the input the exit code is 0; errors: a
// message on standard error, exit code 1 (2: usage).
#include <fstream>
#include <iostream>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "served_model.hpp"

namespace {

using Sequence = cli::ServedModel::Sequence;

struct Options {
  std::string model, out;
  cli::Precision precision = cli::Precision::kDefault;
  int64_t max_tokens = 4096;
};

[[noreturn]] void usage(const char* prog) {
  std::cerr << "usage: " << prog << " --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N]\n";
  std::exit(2);
}

Options parse_options(int argc, char** argv) {
  Options o;
  for (int i = 1; i < argc; ++i) {
    const std::string a = argv[i];
    if (i + 1 >= argc) usage(argv[0]);
    const std::string v = argv[++i];
    if (a == "--model") o.model = v;
    else if (a == "--out") o.out = v;
    else if (a == "--max-tokens") o.max_tokens = std::stoll(v);
    else if (a == "--dtype" && v == "bfloat16") o.precision = cli::Precision::kBf16;
    else if (a == "--dtype" && v == "float32") o.precision = cli::Precision::kFp32;
    else usage(argv[0]);
  }
  if (o.model.empty() || o.out.empty() || o.max_tokens < 1) usage(argv[0]);
  return o;
}

}  // namespace

int main(int argc, char** argv) try {
  const Options opt = parse_options(argc, argv);
  const cli::ServedModel model(opt.model, opt.precision);
  const int64_t V = model.vocab(), cap = opt.max_tokens;
  cudaStream_t stream;
  CUDA_OK(cudaStreamCreate(&stream));
  int64_t* d_ids = nullptr;
  CUDA_OK(cudaMalloc(reinterpret_cast<void**>(&d_ids), static_cast<size_t>(cap) * sizeof(int64_t)));
  float* d_logits = nullptr;
  size_t logits_rows = 0;
  std::vector<float> h_logits;
  std::map<std::string, std::unique_ptr<Sequence>> live;
  std::vector<std::unique_ptr<Sequence>> idle;

  std::string line;
  while (std::getline(std::cin, line)) {
    if (line.find_first_not_of(" \t\r") == std::string::npos) continue;
    const minijson::Value step = minijson::parse(line);
    const long long number = static_cast<long long>(step.at("step").number());
    size_t rows = 0;
    for (const auto& e : step.at("entries").array()) rows += e.at("want").array().size();
    if (rows > logits_rows) {
      cudaFree(d_logits);
      CUDA_OK(cudaMalloc(reinterpret_cast<void**>(&d_logits), rows * V * sizeof(float)));
      logits_rows = rows;
    }
    size_t at = 0;
    for (const auto& e : step.at("entries").array()) {
      std::vector<int64_t> ids;
      std::vector<int32_t> want;
      for (const auto& t : e.at("tokens").array()) ids.push_back(static_cast<int64_t>(t.number()));
      for (const auto& w : e.at("want").array()) want.push_back(static_cast<int32_t>(w.number()));
      if (ids.empty()) throw std::runtime_error("an entry without tokens");
      for (const int64_t id : ids)
        if (id < 0 || id >= V) throw std::runtime_error("token id out of range");
      if (static_cast<int64_t>(ids.size()) > cap) throw std::runtime_error("more tokens than --max-tokens");
      std::unique_ptr<Sequence>& seq = live[e.at("id").string()];
      if (!seq) {
        if (!idle.empty()) {
          seq = std::move(idle.back());
          idle.pop_back();
        } else {
          seq.reset(new Sequence());
          model.make_sequence(cap, seq.get());
        }
      }
      CUDA_OK(cudaMemcpyAsync(d_ids, ids.data(), ids.size() * sizeof(int64_t), cudaMemcpyHostToDevice, stream));
      cli::ctdk_ok(ctdk_decode_extend(seq->decoder, d_ids, static_cast<int64_t>(ids.size()), want.data(),
                                      static_cast<int64_t>(want.size()), want.empty() ? nullptr : d_logits + at * V, stream));
      at += want.size();
    }
    cli::ctdk_ok(ctdk_device_status(stream, nullptr));   // synchronises; a wait that ran out is an error
    if (rows > 0) {
      h_logits.resize(rows * V);
      CUDA_OK(cudaMemcpy(h_logits.data(), d_logits, rows * V * sizeof(float), cudaMemcpyDeviceToHost));
      std::ofstream f(opt.out + "/" + std::to_string(number) + ".f32", std::ios::binary | std::ios::trunc);
      f.write(reinterpret_cast<const char*>(h_logits.data()), static_cast<std::streamsize>(rows * V * sizeof(float)));
      f.close();
      if (!f) throw std::runtime_error("cannot write the logits of step " + std::to_string(number));
    }
    if (step.contains("end"))
      for (const auto& id : step.at("end").array()) {
        auto it = live.find(id.string());
        if (it == live.end()) continue;
        cli::ctdk_ok(ctdk_decode_reset(it->second->decoder, stream));
        idle.push_back(std::move(it->second));
        live.erase(it);
      }
    std::cout << "done " << number << "\n" << std::flush;
  }
  cudaFree(d_logits);
  cudaFree(d_ids);
  return 0;
} catch (const std::exception& e) {
  std::cerr << "[ctd_trace] error: " << e.what() << "\n";
  return 1;
}
