// Decoder of the layer-list family: its buffers and the passes over them. hybrid.cu holds what all layer
// lists share and the sandwich arrangement, hybrid_parallel.cu the parallel arrangement.
#pragma once

#include <functional>
#include <vector>

#include "decode_core.h"
#include "hybrid_kernels.h"
#include "hybrid_model.h"
#include "hybrid_token.h"
#include "parallel_kernels.h"

namespace ctdk {
namespace hybrid {

inline int gemm_rows(const __nv_bfloat16* A, const __nv_bfloat16* W, float* C, int64_t M, int64_t N, int64_t K, int64_t lda,
                     int64_t ldw, int64_t ldc, cudaStream_t s) {
  return ctdk_gemm_bf16(A, W, C, M, N, K, lda, ldw, ldc, s);
}
inline int gemm_rows(const float* A, const float* W, float* C, int64_t M, int64_t N, int64_t K, int64_t lda, int64_t ldw, int64_t ldc,
                     cudaStream_t s) {
  return ctdk_gemm(A, W, C, M, N, K, lda, ldw, ldc, 0, 1, CTDK_GEMM_FP32_SIMT, CTDK_EPI_STORE, nullptr, s);
}

// Device buffers of one branch.
struct BranchBuffers {
  void* cache = nullptr;        // attention
  int64_t chunk = 0;            // cache rows: the chunk, or max_seq when that is smaller
  int rope = -1;                // index of the rotation table
  float* decay = nullptr;       // lightning: per head; then its powers 0 .. 64 per head
  float* powers = nullptr;
  float* state = nullptr;
  float* ring = nullptr;
  void* latent = nullptr;       // latent attention: per position the latent, then the rotated key part
  int64_t ld_latent = 0;
  int64_t n_latent_rot = 0;     // first column of the rotated part
};

struct RopeTable {
  RopeSpec spec;
  int64_t rows = 0;
  float2* table = nullptr;
  double* freqs = nullptr;
};

constexpr int64_t kChunkedRows = 16;   // shorter portions run the recurrences token by token

inline int padded_head(int dim, bool tensor_cores) {
  if (!tensor_cores) return (dim + 3) / 4 * 4;
  return dim <= 64 ? 64 : 128;
}

template <typename T>
struct HybridDecoder : DecoderBase {
  Model m;
  const char* params = nullptr;
  int64_t max_portion = 0;
  std::vector<std::vector<BranchBuffers>> bufs;
  std::vector<RopeTable> ropes;
  float* layers_out = nullptr;

  // prompt-pass buffers, rows = max_portion
  float *x, *proj, *packed, *attn_out, *o32, *y1, *y2, *gu, *dq, *dk, *dv, *dlog, *dbeta, *dz, *dgate;
  T *h, *mixed, *mixed2, *act, *low_a, *low_g;
  float *chunk_state, *cw, *ckh, *cqt, *cu, *cus, *cscores, *cdecay;
  __nv_bfloat16 *qb, *kb, *vb;
  int32_t* want_dev;
  // token-pass buffers
  float *tx[2], *tproj, *tout[2], *tgate, *ty1, *ty2, *tgu, *tpart;
  unsigned int* sync;
  int64_t sync_words = 0;
  TokenPhase* phases_dev;
  std::vector<TokenPhase> phases;
  int stage_floats = 0, token_ctas = 0;
  size_t token_smem = 0;

  template <typename U>
  const U* at(int64_t off) const { return reinterpret_cast<const U*>(params + off); }
  const float* vec(int64_t off) const { return at<float>(off); }
  bool tensor_core_attention(const Branch& b) const { return m.dtype == CTDK_DTYPE_BF16 && b.dim <= 128; }

  bool chunked_lightning(const Branch& b) const { return m.dtype == CTDK_DTYPE_BF16 && lightning_chunked_ok(b.dim, b.vdim); }

  bool chunked_wkv(const Branch& b) const { return m.dtype == CTDK_DTYPE_BF16 && wkv_chunked_ok(b.dim); }

  int carve(Bump& b);
  int build_phases();
  int upload(cudaStream_t s);
  int run_rows(const int64_t* ids, int64_t n, int64_t pos, int64_t done, const int32_t* want, int64_t n_want, float* want_logits,
               bool last, cudaStream_t s);
  int mixer_attention(const Branch& b, const BranchBuffers& bb, int64_t n, int64_t pos, float* y, int64_t ldp, cudaStream_t s);
  int mixer_lightning(const Branch& b, const BranchBuffers& bb, int64_t n, int64_t pos, float* y, int64_t ldp, cudaStream_t s);
  int mixer_delta(const Branch& b, const BranchBuffers& bb, int64_t n, int64_t pos, float* y, int64_t ldp, cudaStream_t s);

  int portion(const int64_t* ids, int64_t n, int64_t pos, const int32_t* want, int64_t n_want, float* want_logits,
              cudaStream_t s) override;
  int token_forward(cudaStream_t s) override;
  int burst(int64_t n, int64_t* out_tokens, cudaStream_t s) override;
  TokenArgs token_args() const;
  int finish_phases();
  int run_head(int64_t n, int64_t done, const int32_t* want, int64_t n_want, float* want_logits, bool last,
               const std::function<int(const int32_t*, int64_t)>& norm, cudaStream_t s);

  // parallel arrangement (hybrid_parallel.cu)
  float *x2, *side, *shift_state, *shift_next;
  T *shifted, *mixes, *low_q, *q_rot, *kv_heads;
  float *q_up, *moe_weight, *expert_gu, *shared_out;
  int32_t *moe_index, *moe_slot, *moe_count, *moe_tiles;
  T *expert_in, *expert_act, *expert_out;
  float *th, *tside, *tq, *tq_abs, *tegu;
  int64_t tside_pitch = 0;   // two side projections, alternating from layer to layer
  int carve_parallel(Bump& b);
  int build_parallel_phases();
  int run_parallel_rows(const int64_t* ids, int64_t n, int64_t pos, int64_t done, const int32_t* want, int64_t n_want,
                        float* want_logits, bool last, cudaStream_t s);
  int mixer_latent(const Layer& L, const BranchBuffers& bb, int64_t n, int64_t pos, cudaStream_t s);
  int mixer_wkv(const Layer& L, const BranchBuffers& bb, int64_t n, int64_t pos, cudaStream_t s);
  int kv_rows(const T* cache, const T* w, int64_t rows, int64_t n, int64_t K, int64_t lda, int64_t ldw, cudaStream_t s);
  int latent_attention(const LatentArgs<T>& a, int64_t pos, int64_t n, cudaStream_t s);
  int feed_forward_rows(const Layer& L, int64_t n, cudaStream_t s);
};

}  // namespace hybrid
}  // namespace ctdk
