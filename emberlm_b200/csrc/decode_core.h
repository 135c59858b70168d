// What every decoder family shares: the position and token counters in device memory, the logits of
// the last position, and the request loop of decode_api.cu (prefill, portions, single steps, greedy
// bursts). A family (decode.cu: the five presets; hybrid.cu: layer-list models) supplies the forward
// passes and owns its caches and recurrent states.
#pragma once

#include "common.cuh"

namespace ctdk {

struct DecoderBase {
  int vocab = 0, max_seq = 0;
  float* logits = nullptr;        // [vocab], device
  int64_t* cur_token = nullptr;   // device: the token a token pass reads
  int* counters = nullptr;        // device: position, tokens generated, scratch, -, 64-bit argmax word
  cudaGraphExec_t graph = nullptr;
  int64_t* graph_out = nullptr;
  cudaStream_t graph_stream = nullptr;
  // Host mirror of the request: tokens run as portions, tokens the greedy loop emitted, tokens fed by step().
  int64_t prompt_len = 0, generated = 0, stepped = 0;

  virtual ~DecoderBase() {
    if (graph != nullptr) cudaGraphExecDestroy(graph);
  }
  // Runs ids[0, T) (device) at positions pos .. pos + T - 1 on the cache and state the positions before
  // left behind (pos == 0: an empty sequence). n_want >= 0: the logits of the rows want[0, n_want)
  // (host, indices into the portion) go to want_logits [n_want, vocab] (device). n_want < 0: those of
  // the last row go to `logits`. Does not touch the counters.
  virtual int portion(const int64_t* ids, int64_t T, int64_t pos, const int32_t* want, int64_t n_want,
                      float* want_logits, cudaStream_t s) = 0;
  // One token pass: *cur_token at position counters[0] -> logits. Does not touch the counters.
  virtual int token_forward(cudaStream_t s) = 0;
  // n greedy tokens in one launch, appended to out_tokens[generated ..], counters advanced. Returns 1
  // when the family has no such kernel for this model (the caller replays token passes).
  virtual int burst(int64_t n, int64_t* out_tokens, cudaStream_t s) = 0;
};

// First index of the maximum as an atomicMax key: floats ordered as unsigned integers in the high
// half, the smaller index preferred in the low half.
__device__ __forceinline__ unsigned long long argmax_key(float v, int idx) {
  unsigned u = __float_as_uint(v);
  u = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
  return (static_cast<unsigned long long>(u) << 32) | (0xFFFFFFFFu - static_cast<unsigned>(idx));
}

// Workspace carving in 256-byte steps; base == nullptr only measures.
struct Bump {
  char* base;
  int64_t used = 0;
  explicit Bump(void* b) : base(static_cast<char*>(b)) {}
  void* bytes(int64_t n) {
    void* p = base ? base + used : nullptr;
    used += (n + 255) / 256 * 256;
    return p;
  }
  float* floats(int64_t n) { return static_cast<float*>(bytes(n * 4)); }
};

#define DTRY(expr)                    \
  do {                                \
    int rc_ = (expr);                 \
    if (rc_ != CTDK_OK) return rc_;   \
  } while (0)

// ---- grid barrier of the persistent token kernels --------------------------------------------
// Barrier words: [0] arrivals, [2] abort flag (all zero at launch).
#ifdef __CUDACC__
__device__ __forceinline__ unsigned int ld_acquire_u32(const unsigned int* p) {
  unsigned int v;
  asm volatile("ld.acquire.gpu.global.u32 %0, [%1];" : "=r"(v) : "l"(p) : "memory");
  return v;
}
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// All CTAs of a cooperative grid meet here: one release reduction on a counter per CTA (no value
// comes back, so the arriving thread does not wait for it; the CTA's earlier writes are ordered
// before it by the bar.sync and the release), then one thread per CTA polls the counter. A flag per
// CTA watched by every other CTA measured twice as slow (all pollers hit the same few L2 lines).
// `epoch` counts the barriers this CTA has passed. Bounded: when the wait runs out, the status word
// gets `where` and the abort flag makes every CTA leave at its next barrier. Returns false once any
// CTA has given up: the caller unwinds.
__device__ __forceinline__ bool grid_barrier(unsigned int* sync, int* status, int where, unsigned int& epoch) {
  __shared__ int s_ok;
  __syncthreads();
  if (threadIdx.x == 0) {
    ++epoch;
    const unsigned int target = epoch * gridDim.x;
    asm volatile("red.release.gpu.global.add.u32 [%0], 1;" ::"l"(&sync[0]) : "memory");
    int ok = 1;
    if (ld_acquire_u32(&sync[0]) < target) {
      const uint64_t t0 = globaltimer_ns();
      unsigned int spins = 0;
      while (ld_acquire_u32(&sync[0]) < target) {
        if ((++spins & 0xffu) == 0u) {
          if (ld_acquire_u32(&sync[2]) != 0u) {   // someone else gave up
            ok = 0;
            break;
          }
          if (globaltimer_ns() - t0 > kWaitBudgetNs) {
            if (atomicCAS(status, 0, CTDK_ETIMEOUT) == 0) {
              status[1] = where;
              status[2] = static_cast<int>(blockIdx.x);
              status[3] = static_cast<int>(epoch);
            }
            atomicExch(&sync[2], 1u);
            ok = 0;
            break;
          }
        }
      }
    }
    if (ok && ld_acquire_u32(&sync[2]) != 0u) ok = 0;
    s_ok = ok;
  }
  __syncthreads();
  return s_ok != 0;
}
#endif

}  // namespace ctdk
