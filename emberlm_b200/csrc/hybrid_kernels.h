// Kernels of the layer-list family, prompt side. Every launcher enqueues on `s` and returns a status.
// T is the model's matrix / activation type (__nv_bfloat16 or float); everything else is fp32.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace ctdk {
namespace hybrid {

// Norm, residual sum, norm in one pass over a row:
//   y   = pending sublayer output (y2 == nullptr), or (rms(y) w_y + rms(y2) w_y2) / 2
//   x   = x + rms(y) w_post              (or, with ids: x = rms(embed[id]) w_embed)
//   h   = rms(x) w_pre, in the model's type, the input of the next projection
// rows of x / y / y2 are gather[i] when gather is given. x_out == nullptr: x is not stored.
template <typename T>
struct NormArgs {
  int width = 0;
  float eps = 0.0f;
  const int64_t* ids = nullptr;
  const T* embed = nullptr;
  int64_t ld_embed = 0;
  const float* w_embed = nullptr;
  const float* x = nullptr;
  const int32_t* gather = nullptr;
  const float *y = nullptr, *y2 = nullptr, *w_y = nullptr, *w_y2 = nullptr, *w_post = nullptr;
  float* x_out = nullptr;
  const float* w_pre = nullptr;
  T* h = nullptr;
  int64_t ld_h = 0;
};
template <typename T>
int norm_rows(const NormArgs<T>& a, int64_t rows, cudaStream_t s);

// act = g sigmoid(1.702 g) (u + 1), g = min(gate, limit), u = clamp(up, +-limit); gu rows hold ffp gate then ffp up columns.
template <typename T>
int clamped_glu_rows(const float* gu, T* act, int64_t rows, int ffp, float limit, cudaStream_t s);

// cos / sin of position * frequency (both in double) for positions [0, n): table[n][pairs].
int rope_table_f64(float2* table, int64_t n, const double* freqs_dev, int pairs, cudaStream_t s);

// ---- chunked attention with tied keys / values ----
// The portion's rows and the cached part of the chunk it starts in, packed for the attention kernels:
// row r holds position chunk_start + r as [H q | G k | G v] heads of Dp columns (columns dim.. zero).
// Rows below `first` come from the cache. Only unrotated keys are cached: they are the values, and
// scores depend on position differences only, so rotating by the place inside the chunk is the same
// as rotating by the absolute position.
template <typename T>
struct AttnArgs {
  const float* proj = nullptr;   // [T rows, ldp] stacked projection
  int64_t ldp = 0;
  int col_q = 0, col_k = 0, col_g = 0;
  const float *b_q = nullptr, *b_k = nullptr;
  int H = 0, G = 0, dim = 0, Dp = 0, rot_pairs = 0;
  int64_t chunk = 0;             // rows of a chunk (= cache rows)
  const float2* table = nullptr; // [chunk, rot_pairs]
  T* cache = nullptr;            // [G][chunk][dim]
  float* packed = nullptr;       // [rows up to a multiple of chunk][(H + 2 G) * Dp]
  float* out = nullptr;          // [same rows][H * Dp]
};
template <typename T>
int attn_pack(const AttnArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s);
// Keys of the last chunk the portion reaches, into the cache (after attn_pack has read it).
template <typename T>
int attn_store(const AttnArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s);
// fp32 attention over the packed rows (any head size): out rows [first, rows).
int attn_chunked_fp32(const float* packed, float* out, int64_t first, int64_t rows, int64_t chunk, int H, int G, int dim, int Dp,
                      float scale, cudaStream_t s);
// dst[t][h * dim + d] = out[first + t][h * Dp + d] * sigmoid(proj[t][col_g + h])
template <typename T>
int attn_gate(const AttnArgs<T>& a, T* dst, int64_t ld, int64_t first, int64_t rows, cudaStream_t s);

// ---- recurrences ----
// State S[H][dim][vdim] (fp32). q / k / v / g are [rows] x heads with the given row pitches; head h reads
// q, k of group h / (H / G). silu != 0: q, k, v pass silu on load. resume == 0: the stored state is
// ignored (a new sequence). Lightning: decay[H]. Delta: logg [rows][H * dim] log decays, beta [rows][H].
// Wkv: decays e^(-e^(z + w0)) from z [rows][ldz] and w0 [H * dim], bonus [H * dim].
enum class Recurrence { kLightning, kDelta, kWkv };
struct ScanArgs {
  const float *q = nullptr, *k = nullptr, *v = nullptr;
  int64_t ldq = 0, ldk = 0, ldv = 0;
  const float* logg = nullptr;
  const float* beta = nullptr;
  const float* decay = nullptr;
  const float *z = nullptr, *w0 = nullptr, *bonus = nullptr;
  int64_t ldz = 0;
  int silu = 0;
  float* state = nullptr;
  float* out = nullptr;   // [rows][H * vdim]
  int H = 0, G = 0, dim = 0, vdim = 0;
  int64_t rows = 0;
  int resume = 0;
};
int recurrent_scan(const ScanArgs& a, Recurrence kind, cudaStream_t s);

// Chunk-parallel lightning attention (bfloat16 models): q, k, v are columns of the projection (before
// silu), powers[h][i] = decay_h^i for i in [0, 64]. Scratch: chunk_state [chunks][H][dk][dv] floats,
// qb / kb [chunks][H][64][dk], vb [chunks][H][64][dv] with dk, dv the tile sizes of lightning_tile().
constexpr int kLightningChunk = 64;
struct LightningArgs {
  const float *q = nullptr, *k = nullptr, *v = nullptr;
  int64_t ldp = 0;
  const float* powers = nullptr;
  float *state = nullptr, *chunk_state = nullptr, *out = nullptr;
  __nv_bfloat16 *qb = nullptr, *kb = nullptr, *vb = nullptr;
  int H = 0, dim = 0, vdim = 0;
  int64_t rows = 0;
  int resume = 0;
};
// Chunk-parallel delta rule: inputs as for recurrent_scan (q, k [rows][G * dim], v [rows][H * vdim], logg
// [rows][H * dim], beta [rows][H], dense). Scratch per (chunk, head), dk / dv the tile sizes: w, kh, qt
// [64][dk], u and us [64][dv], scores [64][64], decay [dk], chunk_state [dk][dv]. split: the products after
// the per-chunk kernel run on the tensor cores with factors of two bfloat16 terms (delta_chunk.cu).
constexpr int kDeltaChunk = 64;
struct DeltaChunkArgs {
  const float *q = nullptr, *k = nullptr, *v = nullptr, *logg = nullptr, *beta = nullptr;
  float *state = nullptr, *out = nullptr;
  float *w = nullptr, *kh = nullptr, *qt = nullptr, *u = nullptr, *us = nullptr, *scores = nullptr, *decay = nullptr, *chunk_state = nullptr;
  int H = 0, G = 0, dim = 0, vdim = 0;
  int64_t rows = 0;
  int resume = 0, split = 0;
};
bool delta_chunked_ok(int dim, int vdim);
int delta_chunked(const DeltaChunkArgs& a, cudaStream_t s);

bool lightning_chunked_ok(int dim, int vdim);
inline int lightning_tile(int d) { return d <= 64 ? 64 : 128; }
int lightning_chunked(const LightningArgs& a, cudaStream_t s);

// rms over all H * vdim columns, * w * sigmoid(gate)
template <typename T>
int gated_norm_rows(const float* o, const float* w, const float* gate, int64_t ldg, T* dst, int64_t ld, int64_t rows, int n, float eps,
                    cudaStream_t s);
// per head: rms over vdim, * w[vdim] * sigmoid(gate)
template <typename T>
int gated_head_norm_rows(const float* o, const float* w, const float* gate, int64_t ldg, T* dst, int64_t ld, int64_t rows, int H,
                         int vdim, float eps, cudaStream_t s);

// What the delta rule reads: convolved, activated, unit-length q and k; v; log decays; beta.
struct DeltaPrepArgs {
  const float* proj = nullptr;
  int64_t ldp = 0;
  int col_q = 0, col_k = 0, col_v = 0, col_b = 0;
  const float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr, *a_log = nullptr, *dt_bias = nullptr;
  const float* z = nullptr;      // [rows][ldz] low-rank decay input W_a2 (W_a1 h)
  int64_t ldz = 0;
  float* ring = nullptr;         // [taps][2 G dim + H vdim]: convolution inputs by position mod taps
  float *q = nullptr, *k = nullptr, *v = nullptr, *logg = nullptr, *beta = nullptr;
  int H = 0, G = 0, dim = 0, vdim = 0, taps = 0;
  int64_t rows = 0, pos = 0;     // first position of the portion
};
int delta_prep(const DeltaPrepArgs& a, cudaStream_t s);
int delta_ring_store(const DeltaPrepArgs& a, cudaStream_t s);

// dst[t][c] = src[t][col + c] in the model's type (inputs of the low-rank second factors)
template <typename T>
int cast_columns(const float* src, int64_t lds, T* dst, int64_t ldd, int64_t rows, int cols, cudaStream_t s);

#ifdef __CUDACC__
__device__ __forceinline__ float sigmoid_f(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x * sigmoid_f(x); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float clamped_glu_f(float gate, float up, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.0f);
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
#endif

}  // namespace hybrid

int attn_chunked_tcgen05(const float* qkv, float* out, int64_t rows, int64_t first, int64_t chunk, int H, int Hk, int D, float scale,
                         cudaStream_t stream);

}  // namespace ctdk
