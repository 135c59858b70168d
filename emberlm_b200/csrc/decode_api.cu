// The request loop shared by every decoder family (decode_core.h): prefill, portions of a prompt,
// single chosen tokens, greedy generation. Token ids and counters stay on the device during greedy
// generation: a burst kernel of the family where it has one, otherwise the token pass captured once
// in a CUDA graph and replayed.
#include "decode_core.h"

namespace ctdk {
namespace {

// First index of the maximum (the reference's greedy sampler, src/core/sampling.cpp:13-20) over
// many CTAs: each reduces its share of the logits and folds (value, index) into one 64-bit word
// with atomicMax (argmax_key); argmax_finish_kernel turns the word into the next input token.
__global__ void __launch_bounds__(256)
    argmax_kernel(const float* __restrict__ logits, int V, unsigned long long* __restrict__ word) {
  __shared__ unsigned long long best_s[8];
  pdl_launch();
  pdl_wait();
  unsigned long long best = 0ull;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < V; i += gridDim.x * blockDim.x) {
    const unsigned long long k = argmax_key(logits[i], i);
    best = k > best ? k : best;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const unsigned long long other = __shfl_xor_sync(0xffffffffu, best, o);
    best = other > best ? other : best;
  }
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  if (lane == 0) best_s[wid] = best;
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int i = 1; i < (blockDim.x >> 5); ++i) best = best_s[i] > best ? best_s[i] : best;
    atomicMax(word, best);
  }
}
// Stores the winning token as the next input, appends it to out_tokens[*count], clears the word and
// advances the counters (pos may point at a scratch int when the position must not move).
__global__ void argmax_finish_kernel(unsigned long long* word, int64_t* cur_token, int64_t* out_tokens, int* pos,
                                     int* count) {
  pdl_launch();
  pdl_wait();
  const int64_t idx = static_cast<int64_t>(0xFFFFFFFFu - static_cast<unsigned>(*word & 0xFFFFFFFFull));
  *cur_token = idx;
  if (out_tokens != nullptr) out_tokens[*count] = idx;
  *word = 0ull;
  *pos += 1;
  *count += 1;
}

__global__ void set_counters_kernel(int* pos, int* count, int p, int c) {
  *pos = p;
  *count = c;
  *reinterpret_cast<unsigned long long*>(pos + 4) = 0ull;   // the argmax word lives behind the counters
}

__global__ void set_token_kernel(int64_t* cur, int* counters, int64_t value, int pos) {
  *cur = value;
  counters[0] = pos;
}
__global__ void place_ids_kernel(int64_t* cur, int* counters, const int64_t* id, int pos) {
  *cur = *id;
  counters[0] = pos;
}

// Position of the next token to be run.
int64_t next_position(const DecoderBase& d) {
  return d.prompt_len + d.stepped + (d.generated > 0 ? d.generated - 1 : 0);
}

int set_counters(DecoderBase& d, int64_t pos, cudaStream_t s) {
  set_counters_kernel<<<1, 1, 0, s>>>(d.counters, d.counters + 1, static_cast<int>(pos), 0);
  return check_launch("decode counters");
}

// One token pass, then the arg-max as the next input token; counters += 1.
int enqueue_token_step(DecoderBase& d, int64_t* out_tokens, cudaStream_t s) {
  DTRY(d.token_forward(s));
  unsigned long long* word = reinterpret_cast<unsigned long long*>(d.counters + 4);
  if (launch_pdl(argmax_kernel, 64, 256, 0, s, d.logits, d.vocab, word) != cudaSuccess)
    return fail(CTDK_ELAUNCH, "decode argmax: launch failed");
  DTRY(check_launch("decode argmax"));
  if (launch_pdl(argmax_finish_kernel, 1, 1, 0, s, word, d.cur_token, out_tokens, d.counters, d.counters + 1) != cudaSuccess)
    return fail(CTDK_ELAUNCH, "decode argmax finish: launch failed");
  return check_launch("decode argmax finish");
}

}  // namespace
}  // namespace ctdk

using namespace ctdk;

extern "C" {

int ctdk_decode_destroy(void* decoder) {
  delete static_cast<DecoderBase*>(decoder);
  return CTDK_OK;
}

int ctdk_decode_reset(void* decoder, void* stream) {
  CTDK_REQUIRE(decoder != nullptr, "ctdk_decode_reset: null decoder");
  DecoderBase& d = *static_cast<DecoderBase*>(decoder);
  d.prompt_len = d.generated = d.stepped = 0;
  return set_counters(d, 0, static_cast<cudaStream_t>(stream));
}

int ctdk_decode_prefill(void* decoder, const int64_t* ids, int64_t T, void* stream) {
  CTDK_REQUIRE(decoder && ids, "ctdk_decode_prefill: null pointer");
  DecoderBase& d = *static_cast<DecoderBase*>(decoder);
  CTDK_REQUIRE(T > 0 && T < d.max_seq, "ctdk_decode_prefill: prompt length must be in [1, max_seq)");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  d.prompt_len = d.generated = d.stepped = 0;
  DTRY(d.portion(ids, T, 0, nullptr, -1, nullptr, s));
  d.prompt_len = T;
  return set_counters(d, T, s);
}

int ctdk_decode_extend(void* decoder, const int64_t* ids, int64_t T, const int32_t* want, int64_t n_want,
                       float* want_logits, void* stream) {
  CTDK_REQUIRE(decoder && ids, "ctdk_decode_extend: null pointer");
  CTDK_REQUIRE(n_want <= 0 || (want && want_logits), "ctdk_decode_extend: wanted rows need an index list and an output");
  DecoderBase& d = *static_cast<DecoderBase*>(decoder);
  CTDK_REQUIRE(d.generated == 0, "ctdk_decode_extend: cannot follow ctdk_decode_greedy; reset or prefill first");
  const int64_t pos = next_position(d);
  CTDK_REQUIRE(T > 0 && pos + T <= d.max_seq, "ctdk_decode_extend: %lld more tokens do not fit into max_seq %d",
               static_cast<long long>(T), d.max_seq);
  for (int64_t i = 0; i < n_want; ++i)
    CTDK_REQUIRE(want[i] >= 0 && want[i] < T, "ctdk_decode_extend: wanted row %lld is not in the portion", static_cast<long long>(i));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (T == 1 && pos > 0) {   // a lone token takes the token pass, as in generation
    place_ids_kernel<<<1, 1, 0, s>>>(d.cur_token, d.counters, ids, static_cast<int>(pos));
    DTRY(check_launch("decode place token"));
    DTRY(d.token_forward(s));
    for (int64_t i = 0; i < n_want; ++i)
      if (cudaMemcpyAsync(want_logits + i * d.vocab, d.logits, sizeof(float) * d.vocab, cudaMemcpyDeviceToDevice, s) != cudaSuccess)
        return fail(CTDK_ELAUNCH, "ctdk_decode_extend: copying the logits failed");
  } else {
    DTRY(d.portion(ids, T, pos, want, n_want, want_logits, s));
  }
  d.prompt_len += T;
  return set_counters(d, pos + T, s);
}

int ctdk_decode_logits(void* decoder, const float** logits) {
  CTDK_REQUIRE(decoder && logits, "ctdk_decode_logits: null pointer");
  *logits = static_cast<DecoderBase*>(decoder)->logits;
  return CTDK_OK;
}

int ctdk_decode_step(void* decoder, int64_t token, void* stream) {
  CTDK_REQUIRE(decoder != nullptr, "ctdk_decode_step: null decoder");
  DecoderBase& d = *static_cast<DecoderBase*>(decoder);
  CTDK_REQUIRE(d.prompt_len > 0, "ctdk_decode_step: call ctdk_decode_prefill first");
  CTDK_REQUIRE(d.generated == 0, "ctdk_decode_step: cannot be mixed with ctdk_decode_greedy after one prefill");
  CTDK_REQUIRE(token >= 0 && token < d.vocab, "ctdk_decode_step: token id out of range");
  const int64_t pos = next_position(d);
  CTDK_REQUIRE(pos < d.max_seq, "ctdk_decode_step: the cache is full (max_seq %d)", d.max_seq);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  set_token_kernel<<<1, 1, 0, s>>>(d.cur_token, d.counters, token, static_cast<int>(pos));
  DTRY(check_launch("decode set token"));
  DTRY(d.token_forward(s));
  ++d.stepped;
  return set_counters(d, pos + 1, s);
}

int ctdk_decode_greedy(void* decoder, int64_t n_new, int64_t* out_tokens, void* stream) {
  CTDK_REQUIRE(decoder && out_tokens, "ctdk_decode_greedy: null pointer");
  CTDK_REQUIRE(n_new >= 0, "ctdk_decode_greedy: negative token count");
  DecoderBase& d = *static_cast<DecoderBase*>(decoder);
  CTDK_REQUIRE(d.prompt_len > 0, "ctdk_decode_greedy: call ctdk_decode_prefill first");
  CTDK_REQUIRE(d.stepped == 0, "ctdk_decode_greedy: cannot be mixed with ctdk_decode_step after one prefill");
  // n tokens after the prompt need n - 1 cache positions (the first comes from the prompt's logits, the
  // last is not fed back): the reference's loop emits max_seq - prompt + 1 tokens before it reports
  // max_seq_len (tools/ctd_generate/main.cpp:143-179)
  CTDK_REQUIRE(d.prompt_len + d.generated + n_new <= d.max_seq + 1,
               "ctdk_decode_greedy: %lld more tokens would exceed max_seq %d", static_cast<long long>(n_new),
               d.max_seq);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int64_t todo = n_new;
  if (todo > 0 && d.generated == 0) {
    // the first new token comes from the prefill logits; its position is the prompt length
    unsigned long long* word = reinterpret_cast<unsigned long long*>(d.counters + 4);
    argmax_kernel<<<64, 256, 0, s>>>(d.logits, d.vocab, word);
    DTRY(check_launch("decode argmax"));
    // count += 1; the position is unchanged (a scratch int takes the increment)
    argmax_finish_kernel<<<1, 1, 0, s>>>(word, d.cur_token, out_tokens, d.counters + 2, d.counters + 1);
    DTRY(check_launch("decode argmax finish"));
    d.generated = 1;
    --todo;
  }
  if (todo == 0) return CTDK_OK;
  // All remaining tokens in one launch where the family has a burst kernel for this model.
  {
    const int rc = d.burst(todo, out_tokens, s);
    if (rc <= 0) {
      if (rc == CTDK_OK) d.generated += todo;
      return rc;
    }
  }
  // One token step = ~9 kernels per layer; captured once and replayed, so a step costs one launch.
  const bool can_capture = s != nullptr;
  if (can_capture && (d.graph == nullptr || d.graph_out != out_tokens || d.graph_stream != s)) {
    if (d.graph != nullptr) {
      cudaGraphExecDestroy(d.graph);
      d.graph = nullptr;
    }
    cudaGraph_t g = nullptr;
    cudaError_t e = cudaStreamBeginCapture(s, cudaStreamCaptureModeThreadLocal);
    if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "decode: begin capture: %s", cudaGetErrorString(e));
    const int rc = enqueue_token_step(d, out_tokens, s);
    e = cudaStreamEndCapture(s, &g);
    if (rc != CTDK_OK) {
      if (g != nullptr) cudaGraphDestroy(g);
      return rc;
    }
    if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "decode: end capture: %s", cudaGetErrorString(e));
    e = cudaGraphInstantiate(&d.graph, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "decode: graph instantiate: %s", cudaGetErrorString(e));
    d.graph_out = out_tokens;
    d.graph_stream = s;
  }
  for (int64_t i = 0; i < todo; ++i) {
    if (can_capture) {
      cudaError_t e = cudaGraphLaunch(d.graph, s);
      if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "decode: graph launch: %s", cudaGetErrorString(e));
    } else {
      DTRY(enqueue_token_step(d, out_tokens, s));
    }
  }
  d.generated += todo;
  return CTDK_OK;
}

}  // extern "C"
