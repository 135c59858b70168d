// A model as the serving tools use it: found on disk, weights in device memory, decoders made from it.
// Two families:
//   presets      a safetensors file (or a folder with model.safetensors whose config.json names no
//                layer-list architecture): one of the five architectures of model_desc.hpp, recognised
//                by the shape of its embedding;
//   layer lists  a folder whose config.json has an "architecture" that ctdk_hybrid_open knows.
// A build without the presets (CTD_WITH_PRESETS=0) serves layer lists only and needs none of the
// training-path kernels.
#pragma once

#include <sys/stat.h>

#include <cstdint>
#include <cstring>
#include <fstream>
#include <sstream>
#include <stdexcept>
#include <string>
#include <vector>

#include <cuda_runtime.h>

#include "../../include/ctdk.h"
#include "../../include/ctdk_util/minijson.hpp"
#include "../../include/ctdk_util/safetensors.hpp"
#ifndef CTD_WITH_PRESETS
#define CTD_WITH_PRESETS 1
#endif
#if CTD_WITH_PRESETS
#include "model_desc.hpp"
#endif

namespace cli {

inline void cuda_ok(cudaError_t e, const char* what) {
  if (e != cudaSuccess) throw std::runtime_error(std::string(what) + ": " + cudaGetErrorString(e));
}
inline void ctdk_ok(int rc) {
  if (rc != CTDK_OK) throw std::runtime_error(std::string(ctdk_last_error()));
}
#define CUDA_OK(expr) ::cli::cuda_ok((expr), #expr)

// Arithmetic of a served model. kDefault: what the family serves with (presets: fp32 prompt products;
// layer lists: bfloat16).
enum class Precision { kDefault, kBf16, kTf32, kFp32 };

class ServedModel {
 public:
  ServedModel(const std::string& path, Precision precision) {
    struct stat st;
    const bool dir = stat(path.c_str(), &st) == 0 && S_ISDIR(st.st_mode);
    std::string config;
    if (dir) {
      std::ifstream in(path + "/config.json");
      std::ostringstream text;
      text << in.rdbuf();
      if (in) config = text.str();
    }
    st::File file(dir ? path + "/model.safetensors" : path);
    if (!config.empty() && minijson::parse(config).contains("architecture")) open_layer_list(config, file, precision);
    else open_preset(file, precision);
  }
  ServedModel(const ServedModel&) = delete;
  ServedModel& operator=(const ServedModel&) = delete;
  ~ServedModel() {
    if (hybrid_ != nullptr) ctdk_hybrid_close(hybrid_);
    cudaFree(params_);
  }

  int64_t vocab() const { return vocab_; }
  const std::string& summary() const { return summary_; }

  // A decoder with its own workspace for one live sequence of at most max_seq tokens.
  struct Sequence {
    void* decoder = nullptr;
    void* workspace = nullptr;
    Sequence() = default;
    Sequence(const Sequence&) = delete;
    Sequence& operator=(const Sequence&) = delete;
    ~Sequence() {
      if (decoder != nullptr) ctdk_decode_destroy(decoder);
      cudaFree(workspace);
    }
  };
  void make_sequence(int64_t max_seq, Sequence* out) const {
    const int64_t portion = max_seq < kPortion ? max_seq : kPortion;
    int64_t bytes = -1;
    if (hybrid_ != nullptr) bytes = ctdk_hybrid_workspace_bytes(hybrid_, max_seq, portion);
#if CTD_WITH_PRESETS
    else bytes = ctdk_decode_workspace_bytes(&preset_, max_seq);
#endif
    if (bytes < 0) throw std::runtime_error(ctdk_last_error());
    CUDA_OK(cudaMalloc(&out->workspace, static_cast<size_t>(bytes)));
    if (hybrid_ != nullptr) ctdk_ok(ctdk_hybrid_decode_create(hybrid_, params_, out->workspace, bytes, max_seq, portion, &out->decoder));
#if CTD_WITH_PRESETS
    else ctdk_ok(ctdk_decode_create(&preset_, static_cast<const float*>(params_), out->workspace, bytes, max_seq, &out->decoder));
#endif
  }

 private:
  static constexpr int64_t kPortion = 4096;   // rows of a layer-list prompt run at once
  void* hybrid_ = nullptr;
  void* params_ = nullptr;
  int64_t vocab_ = 0;
  std::string summary_;
#if CTD_WITH_PRESETS
  ctdk_model_config preset_{};
#endif

  void upload(const void* host, size_t bytes) {
    CUDA_OK(cudaSetDevice(0));
    CUDA_OK(cudaMalloc(&params_, bytes));
    CUDA_OK(cudaMemcpy(params_, host, bytes, cudaMemcpyHostToDevice));
  }

  void open_layer_list(const std::string& config, st::File& file, Precision precision) {
    if (precision == Precision::kTf32) throw std::runtime_error("layer-list models run in bf16 or fp32");
    const int dtype = precision == Precision::kFp32 ? CTDK_DTYPE_F32 : CTDK_DTYPE_BF16;
    ctdk_ok(ctdk_hybrid_open(config.c_str(), file.header_text().c_str(), dtype, &hybrid_));
    vocab_ = ctdk_hybrid_vocab(hybrid_);
    std::vector<unsigned char> arena(static_cast<size_t>(ctdk_hybrid_arena_bytes(hybrid_)), 0);
    const int64_t n = ctdk_hybrid_num_tensors(hybrid_);
    std::vector<float> f;
    std::vector<uint16_t> raw;
    for (int64_t i = 0; i < n; ++i) {
      ctdk_tensor_info t;
      ctdk_ok(ctdk_hybrid_tensor(hybrid_, i, &t));
      const int64_t count = t.rows * t.cols;
      const bool bf16 = file.entry(t.name).dtype == "BF16";
      f.resize(count);
      raw.resize(count);
      if (bf16) {
        file.read_bf16(t.name, raw.data(), count);
        for (int64_t k = 0; k < count; ++k) f[k] = widen(raw[k]);
      } else {
        file.read_f32(t.name, f.data(), count);
        for (int64_t k = 0; k < count; ++k) raw[k] = round_bf16(f[k]);
      }
      for (int64_t r = 0; r < t.rows; ++r) {
        if (t.is_matrix && dtype == CTDK_DTYPE_BF16)
          std::memcpy(arena.data() + t.offset + r * t.ld * 2, raw.data() + r * t.cols, t.cols * 2);
        else
          std::memcpy(arena.data() + t.offset + r * t.ld * 4, f.data() + r * t.cols, t.cols * 4);
      }
    }
    upload(arena.data(), arena.size());
    summary_ = "layer list, " + std::to_string(n) + " tensors, vocab " + std::to_string(vocab_) +
               (dtype == CTDK_DTYPE_BF16 ? ", bf16" : ", fp32");
  }

  void open_preset(st::File& file, Precision precision) {
#if CTD_WITH_PRESETS
    if (precision == Precision::kBf16) precision = Precision::kTf32;   // the 16-bit request's nearest: TF32 prompt products
    const st::Entry& emb = file.entry("model.embed_tokens.weight");
    if (emb.shape.size() != 2) throw std::runtime_error("autodetect_config: model.embed_tokens.weight must be 2-D");
    preset_ = autodetect_config(emb.shape[0], emb.shape[1]);
    preset_.precision = precision == Precision::kTf32 ? CTDK_GEMM_TF32 : CTDK_GEMM_3XTF32;
    vocab_ = preset_.vocab_size;
    int64_t floats = 0;
    const std::vector<ParamDesc> params = describe_parameters(preset_, &floats);
    std::vector<float> arena(static_cast<size_t>(floats), 0.0f);
    for (const auto& p : params) file.read_f32(p.name, arena.data() + p.offset, p.numel);
    upload(arena.data(), arena.size() * sizeof(float));
    summary_ = "hidden=" + std::to_string(preset_.hidden_size) + " layers=" + std::to_string(preset_.num_hidden_layers);
#else
    (void)file;
    (void)precision;
    throw std::runtime_error("this build serves layer-list models only");
#endif
  }

  static float widen(uint16_t v) {
    const uint32_t u = static_cast<uint32_t>(v) << 16;
    float f;
    std::memcpy(&f, &u, 4);
    return f;
  }
  static uint16_t round_bf16(float f) {   // to nearest, ties to even
    uint32_t u;
    std::memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return static_cast<uint16_t>((u >> 16) | 0x40u);
    return static_cast<uint16_t>((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
  }
};

}  // namespace cli
