// Kernels of the parallel arrangement's prompt pass: residual with gated sublayers, grouped norm, token
// shift; latent attention; time mixing with a bonus (wkv); mixture of experts. Every launcher enqueues on
// `s` and returns a status. T is the model's matrix / activation type; everything else is fp32.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace ctdk {
namespace hybrid {

// One pass over the rows of a portion:
//   x  = ids ? embed[id] * scale : x + sigmoid(z1 + b1) y1 + sigmoid(z2 + b2) y2      (y2 may be null)
//   h  = w * x with every group of width / groups columns divided by its root mean square
//   m  = h + (previous row's h - h) * shift                                          (shift may be null)
//   mix[i] = m + (previous row's m - m) * mu[i]                                      (n_mix may be 0)
// h, m and the mixes are stored in the model's type; the previous row of row 0 is prev_h / prev_m (null:
// zeros), the last row's go to next_h / next_m in fp32. Rows are gather[i] when gather is given (no shift
// then). x and x_out must not overlap; x_out may be null.
constexpr int kMaxMixes = 5;
template <typename T>
struct ShiftNormArgs {
  int width = 0, groups = 1, n_mix = 0;
  float eps = 0.0f, scale = 1.0f;
  const int64_t* ids = nullptr;
  const T* embed = nullptr;
  int64_t ld_embed = 0;
  const float* x = nullptr;
  const float *y1 = nullptr, *y2 = nullptr, *z1 = nullptr, *z2 = nullptr, *b1 = nullptr, *b2 = nullptr;
  int64_t ldz = 0;
  const int32_t* gather = nullptr;
  float* x_out = nullptr;
  const float *w = nullptr, *shift = nullptr, *mu[kMaxMixes] = {};
  T *h = nullptr, *shifted = nullptr, *mix = nullptr;
  int64_t ld_h = 0, mix_stride = 0;   // elements between two mixes
  const float *prev_h = nullptr, *prev_m = nullptr;
  float *next_h = nullptr, *next_m = nullptr;
};
template <typename T>
int shift_norm_rows(const ShiftNormArgs<T>& a, int64_t rows, cudaStream_t s);
// state[layer][slot][2][width] = next[layer][2][width]
int commit_shift_state(const float* next, float* state, int layers, int slot, int width, cudaStream_t s);

// act = f(gate) * up for rows of ffp gate then ffp up columns; rows_dev (may be null): a device count that
// caps `rows`.
enum class Glu { kSilu, kGelu };
template <typename T>
int glu_rows(const float* gu, int64_t ldg, T* act, int64_t lda, int64_t rows, int ffp, Glu kind, const int32_t* rows_dev, cudaStream_t s);

// ---- latent attention ----
// Cached row of a position: kv_rank latent columns (zero up to rot_col), rot_dim rotated key columns.
template <typename T>
struct LatentArgs {
  const float* proj = nullptr;        // [rows, ldp]: q_rank, kv_rank + rot_dim and heads columns at col_q, col_k, col_g
  int64_t ldp = 0;
  int col_q = 0, col_k = 0, col_g = 0;
  int H = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, q_rank = 0;
  float eps = 0.0f, scale = 0.0f;
  const float *q_norm = nullptr, *kv_norm = nullptr;
  const float2* table = nullptr;      // [max_seq, rot_dim / 2]
  T* cache = nullptr;                 // [max_seq, ld_cache]
  int64_t ld_cache = 0;
  int rot_col = 0;
  T* low_q = nullptr;                 // [rows, ld_low]
  int64_t ld_low = 0;
  const float* q_up = nullptr;        // [rows, ld_up] queries, heads of dim + rot_dim
  int64_t ld_up = 0;
  T* q = nullptr;                     // [rows, H, pad8(dim) + pad8(rot_dim)] rotated
  const T* kv = nullptr;              // [first + rows, ld_kv]: H * dim key columns, from col_v on H * vdim value columns
  int64_t ld_kv = 0;
  int col_v = 0;
  T* out = nullptr;                   // [rows, ld_out] gated
  int64_t ld_out = 0;
};
inline __host__ __device__ int latent_q_pitch(int dim, int rot_dim) { return (dim + 7) / 8 * 8 + (rot_dim + 7) / 8 * 8; }
// Norms of the two down projections, rotation of the shared key part: low_q and the cache rows first ...
template <typename T>
int latent_prep(const LatentArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s);
// Rotation of the queries: q_up -> q.
template <typename T>
int latent_rotate(const LatentArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s);
// Causal attention of the portion's rows over all positions so far, gated; fp32 arithmetic, any size.
template <typename T>
int latent_attention_fp32(const LatentArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s);
// The same on the tensor cores (bfloat16 operands); sizes it takes.
bool latent_tcgen05_ok(int dim, int rot_dim, int vdim);
int latent_attention_tcgen05(const LatentArgs<__nv_bfloat16>& a, int64_t first, int64_t rows, cudaStream_t s);

// ---- time mixing ----
// dst[t][c] = tanh(src[t][c]), zero up to ldd
template <typename T>
int tanh_rows(const float* src, int64_t lds, T* dst, int64_t ldd, int64_t rows, int n, cudaStream_t s);
// Chunk-parallel form for bfloat16 models (wkv_chunk.cu), up to the gated norm: r, k, v, gate are columns of
// the projection, decays e^(-e^(z + w0)). Scratch, with d = wkv_tile(dim): chunk_state [chunks][H][d][d],
// decay [chunks][H][d].
constexpr int kWkvChunk = 64;
struct WkvArgs {
  const float *r = nullptr, *k = nullptr, *v = nullptr, *gate = nullptr;
  int64_t ldp = 0;
  const float *z = nullptr, *w0 = nullptr, *bonus = nullptr, *w_norm = nullptr;
  int64_t ldz = 0;
  float *state = nullptr, *chunk_state = nullptr, *decay = nullptr;
  __nv_bfloat16* out = nullptr;
  int64_t ld_out = 0;
  int H = 0, dim = 0;
  float eps = 0.0f;
  int64_t rows = 0;
  int resume = 0;
};
inline int wkv_tile(int dim) { return dim <= 64 ? 64 : 128; }
bool wkv_chunked_ok(int dim);
int wkv_chunked(const WkvArgs& a, cudaStream_t s);
// per head: rms over dim, * w[head * dim ..] * silu(gate)
template <typename T>
int silu_head_norm_rows(const float* o, const float* w, const float* gate, int64_t ldg, T* dst, int64_t ld, int64_t rows, int H, int dim,
                        float eps, cudaStream_t s);

// ---- mixture of experts ----
// Routing of a portion: chosen outputs [rows][top] with weights, then one slot per chosen expert. Slots of an
// expert are consecutive and start at a multiple of kMoeTile; tiles[i] is the expert of slots
// [i * kMoeTile, ..), tiles[max_tiles] their number; slot -1: an identity output.
constexpr int kMoeTile = 128;
struct MoeArgs {
  const float* z = nullptr;           // [rows, ldz] router logits
  int64_t ldz = 0;
  const float* correction = nullptr;
  int experts = 0, outputs = 0, top = 0, groups = 1, keep = 1;
  int32_t *index = nullptr, *slot = nullptr;    // [rows][top]
  float* weight = nullptr;                      // [rows][top]
  int32_t* count = nullptr;                     // [2][experts]: rows per expert, first slot of each
  int32_t* tiles = nullptr;                     // [max_tiles + 2]: expert per tile, number of tiles, number of slots
  int max_tiles = 0;
};
inline int64_t moe_max_tiles(int64_t rows, int experts, int top) {
  const int64_t n = rows * top;
  return n / kMoeTile + (n < experts ? n : experts);
}
int moe_route(const MoeArgs& a, int64_t rows, cudaStream_t s);
// xe[slot] = h[row]
template <typename T>
int moe_gather(const MoeArgs& a, const T* h, int64_t ld_h, T* xe, int width, int64_t rows, cudaStream_t s);
// act[slot] = silu(gate) up of the slot's expert: 2 * effp rows of w per expert (gate rows, then up rows), K
// columns. scratch (fp32 models): [slots, 2 * effp].
int experts_up(const MoeArgs& a, const float* xe, int64_t ld_x, const float* w, int64_t ldw, int K, int effp, float* act, float* scratch,
               cudaStream_t s);
int experts_up(const MoeArgs& a, const __nv_bfloat16* xe, int64_t ld_x, const __nv_bfloat16* w, int64_t ldw, int K, int effp,
               __nv_bfloat16* act, float* scratch, cudaStream_t s);
// out[slot] = the down product of the slot's expert: n_pitch rows of w per expert, of which N count, K columns.
int experts_down(const MoeArgs& a, const float* act, int64_t ld_a, const float* w, int64_t ldw, int64_t n_pitch, int N, int K, float* out,
                 int64_t ld_out, cudaStream_t s);
int experts_down(const MoeArgs& a, const __nv_bfloat16* act, int64_t ld_a, const __nv_bfloat16* w, int64_t ldw, int64_t n_pitch, int N, int K,
                 __nv_bfloat16* out, int64_t ld_out, cudaStream_t s);
// y[row] = sum weight * (expert_out[slot] or h[row]) + sigmoid(sg) * shared
template <typename T>
int moe_combine(const MoeArgs& a, const T* expert_out, int64_t ld_eo, const T* h, int64_t ld_h, const float* sg, int64_t ld_sg,
                const float* shared, float* y, int width, int64_t rows, cudaStream_t s);

#ifdef __CUDACC__
__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
#endif

}  // namespace hybrid
}  // namespace ctdk
