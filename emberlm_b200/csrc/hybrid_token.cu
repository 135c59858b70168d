// Persistent token kernel of the layer-list family (hybrid_token.h). Per layer with two branches:
//   [sandwich norms + stacked input projection] | [mix: attention key ranges, recurrent heads]
//   | [branch norms and gates + output projections] | [branch average, norms + gate|up] | [GLU + down]
// and per token the head with the arg-max. A cooperative grid stays resident over all tokens of a
// launch; every phase deals its rows (or its heads) to the CTAs, and while a CTA waits at a barrier
// the weights of a coming phase are on their way into L2. Vectors between phases are fp32; every CTA
// stages (and norms) its own copy. All waits are bounded.
//
// Phases of the parallel arrangement (kStageList; a kernel of its own with one CTA of 16 warps per SM) are
// more uniform: operations that fill the staged vector, up to six products reading parts of it, and the
// items of a mixer (recurrent heads, ranges of the latent cache). The feed-forward's products ride along in
// the mixer's phases: per latent-attention layer
//   [norm, shift + every projection] | [queries, choice of the experts + their gate / up rows]
//   | [queries against the cache rows + down rows] | [ranges of the cache] | [merge, values] | [output]
// and for time mixing [norm, shift, mixes + projections] | [state + experts' rows] | [output + down rows].
#include <cfloat>
#include <type_traits>

#include "decode_core.h"
#include "hybrid_kernels.h"
#include "hybrid_token.h"
#include "mma_bf16.cuh"
#include "moe_route.cuh"
#include "parallel_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int kThreads = 256, kWarps = 8;
constexpr int token_threads(bool list) { return list ? kListThreads : kThreads; }

__device__ __forceinline__ float ldg_f(const float* p) { return __ldcg(p); }

// Eight (bfloat16) or four (fp32) weights against the staged vector.
template <typename T>
struct Chunk;
template <>
struct Chunk<float> {
  static constexpr int kN = 4;
  float4 w;
  __device__ __forceinline__ void load(const float* p) { w = __ldcs(reinterpret_cast<const float4*>(p)); }
  __device__ __forceinline__ float dot(const float* x, float acc) const {
    const float4 v = *reinterpret_cast<const float4*>(x);
    acc = fmaf(w.x, v.x, acc);
    acc = fmaf(w.y, v.y, acc);
    acc = fmaf(w.z, v.z, acc);
    return fmaf(w.w, v.w, acc);
  }
  __device__ __forceinline__ void unpack(float (&o)[4]) const {
    o[0] = w.x;
    o[1] = w.y;
    o[2] = w.z;
    o[3] = w.w;
  }
};
template <>
struct Chunk<__nv_bfloat16> {
  static constexpr int kN = 8;
  uint4 w;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { w = __ldcs(reinterpret_cast<const uint4*>(p)); }
  __device__ __forceinline__ float dot(const float* x, float acc) const {
    const float4 a = *reinterpret_cast<const float4*>(x), b = *reinterpret_cast<const float4*>(x + 4);
    acc = fmaf(__uint_as_float(w.x << 16), a.x, acc);
    acc = fmaf(__uint_as_float(w.x & 0xffff0000u), a.y, acc);
    acc = fmaf(__uint_as_float(w.y << 16), a.z, acc);
    acc = fmaf(__uint_as_float(w.y & 0xffff0000u), a.w, acc);
    acc = fmaf(__uint_as_float(w.z << 16), b.x, acc);
    acc = fmaf(__uint_as_float(w.z & 0xffff0000u), b.y, acc);
    acc = fmaf(__uint_as_float(w.w << 16), b.z, acc);
    return fmaf(__uint_as_float(w.w & 0xffff0000u), b.w, acc);
  }
  __device__ __forceinline__ void unpack(float (&o)[8]) const {
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      o[2 * i] = __uint_as_float(u[i] << 16);
      o[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
  }
};

// dot(W[row, part of K], xs) over a warp that owns the chunks part, part + WPR, ...: the lane's share of the sum.
template <typename T>
__device__ __forceinline__ float row_part(const T* __restrict__ row, const float* xs, int K, int part, int wpr) {
  constexpr int N = Chunk<T>::kN;
  const int lane = threadIdx.x & 31;
  const int n = K / N, step = 32 * wpr;
  float acc = 0.0f;
  int i = part * 32 + lane;
  for (; i + 3 * step < n; i += 4 * step) {
    Chunk<T> c[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) c[u].load(row + static_cast<int64_t>(i + u * step) * N);
#pragma unroll
    for (int u = 0; u < 4; ++u) acc = c[u].dot(xs + (i + u * step) * N, acc);
  }
  for (; i < n; i += step) {
    Chunk<T> c;
    c.load(row + static_cast<int64_t>(i) * N);
    acc = c.dot(xs + i * N, acc);
  }
  return acc;
}
// All lanes get the sum.
template <typename T>
__device__ __forceinline__ float row_dot(const T* __restrict__ row, const float* xs, int K, int part, int wpr) {
  return warp_sum(row_part<T>(row, xs, K, part, wpr));
}

template <int N>
__device__ __forceinline__ void block_sum(float (&v)[N], float* red /* [N][8] */) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  __syncthreads();
#pragma unroll
  for (int k = 0; k < N; ++k) {
    v[k] = warp_sum(v[k]);
    if (lane == 0) red[k * kWarps + wid] = v[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < N; ++k) {
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < kWarps; ++i) t += red[k * kWarps + i];
    v[k] = t;
  }
}

// xs[0, width) = the normed input of a projection; CTA 0 stores the new residual. Zero padding to a multiple of 8.
template <typename T>
__device__ void stage_norm(const TokenArgs& a, const TokenPhase& ph, int64_t tok, float* xs, float* red) {
  const int W = a.width;
  const float inv = 1.0f / static_cast<float>(W);
  float ss[2] = {0.0f, 0.0f};
  // a thread keeps to its own columns until the last barrier
  if (ph.first_token) {
    const T* e = static_cast<const T*>(a.embed) + tok * a.ld_embed;
    for (int i = threadIdx.x; i < W; i += kThreads) {
      const float v = to_f(e[i]);
      xs[i] = v;
      ss[0] += v * v;
    }
    block_sum<2>(ss, red);
    const float sc = rsqrtf(ss[0] * inv + a.eps);
    for (int i = threadIdx.x; i < W; i += kThreads) xs[i] *= sc * a.w_embed[i];
  } else {
    if (ph.y2 != nullptr) {
      for (int i = threadIdx.x; i < W; i += kThreads) {
        const float u = ldg_f(ph.y + i), v = ldg_f(ph.y2 + i);
        ss[0] += u * u;
        ss[1] += v * v;
      }
      block_sum<2>(ss, red);
      const float s1 = rsqrtf(ss[0] * inv + a.eps), s2 = rsqrtf(ss[1] * inv + a.eps);
      ss[0] = ss[1] = 0.0f;
      for (int i = threadIdx.x; i < W; i += kThreads) {
        const float v = 0.5f * (ldg_f(ph.y + i) * s1 * ph.w_y[i] + ldg_f(ph.y2 + i) * s2 * ph.w_y2[i]);
        xs[i] = v;
        ss[0] += v * v;
      }
    } else {
      for (int i = threadIdx.x; i < W; i += kThreads) {
        const float v = ldg_f(ph.y + i);
        xs[i] = v;
        ss[0] += v * v;
      }
    }
    block_sum<2>(ss, red);
    const float sc = rsqrtf(ss[0] * inv + a.eps);
    for (int i = threadIdx.x; i < W; i += kThreads) xs[i] = ldg_f(ph.x + i) + xs[i] * sc * ph.w_post[i];
  }
  ss[0] = ss[1] = 0.0f;
  for (int i = threadIdx.x; i < W; i += kThreads) {
    const float v = xs[i];
    if (blockIdx.x == 0 && ph.x_out != nullptr) ph.x_out[i] = v;
    ss[0] += v * v;
  }
  block_sum<2>(ss, red);
  const float sc = rsqrtf(ss[0] * inv + a.eps);
  for (int i = threadIdx.x; i < W; i += kThreads) xs[i] *= sc * ph.w_pre[i];
  if (threadIdx.x < 8 && W + threadIdx.x < ((W + 7) & ~7)) xs[W + threadIdx.x] = 0.0f;
  __syncthreads();
}

// Outputs of the mix phase as inputs of the output projections.
__device__ void stage_mixed(const TokenArgs& a, const TokenPhase& ph, float* sm, float* red) {
  for (int b = 0; b < ph.n_branch; ++b) {
    const TokenBranch& br = ph.br[b];
    float* xs = sm + br.stage_at;
    const int n = br.H * br.vdim;
    if (br.kind == kTokAttention) {
      for (int i = threadIdx.x; i < n; i += kThreads) xs[i] = ldg_f(br.out + i);
    } else if (br.kind == kTokLightning) {
      float ss[1] = {0.0f};
      for (int i = threadIdx.x; i < n; i += kThreads) {
        const float v = ldg_f(br.out + i);
        xs[i] = v;
        ss[0] += v * v;
      }
      block_sum<1>(ss, red);
      const float sc = rsqrtf(ss[0] / static_cast<float>(n) + a.eps);
      for (int i = threadIdx.x; i < n; i += kThreads) xs[i] *= sc * br.w_norm[i] * sigmoid_f(ldg_f(ph.proj + br.col_g + i));
    } else {
      const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
      for (int h = wid; h < br.H; h += kWarps) {
        float ss = 0.0f;
        for (int d = lane; d < br.vdim; d += 32) {
          const float v = ldg_f(br.out + h * br.vdim + d);
          ss += v * v;
        }
        const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(br.vdim) + a.eps);
        for (int d = lane; d < br.vdim; d += 32)
          xs[h * br.vdim + d] = ldg_f(br.out + h * br.vdim + d) * sc * br.w_norm[d] * sigmoid_f(ldg_f(br.gate + h * br.vdim + d));
      }
    }
    if (threadIdx.x < 8 && n + threadIdx.x < ((n + 7) & ~7)) xs[n + threadIdx.x] = 0.0f;
  }
  __syncthreads();
}

// Attention of the new token over one key range of key/value head g, all query heads of the group;
// the range that arrives last merges them and applies the head gates.
template <typename T>
__device__ void attention_item(const TokenPhase& ph, const TokenBranch& br, int item, int pos, float* sm, int* s_flag) {
  const int g = item / kAttnSplits, sp = item % kAttnSplits;
  const int dim = br.dim, hq = br.H / br.G, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int slot = pos % br.chunk, L = slot + 1;
  int n_act = (L + 31) / 32;
  if (n_act > kAttnSplits) n_act = kAttnSplits;
  const int per = (L + n_act - 1) / n_act;
  n_act = (L + per - 1) / per;
  if (sp >= n_act) return;
  const int j0 = sp * per, j1 = min(L, j0 + per);
  const int KT = dim <= 128 ? 32 : (dim <= 256 ? 16 : (dim <= 512 ? 8 : 4)), ldk = dim + 1;
  float* qs = sm;                        // [hq][dim] rotated, scaled
  float* kr = qs + hq * dim;             // [KT][ldk] keys = values
  float* kt = kr + KT * ldk;             // [KT][ldk] rotated keys
  float* sc = kt + KT * ldk;             // [hq][32]
  float* st = sc + hq * 32;              // [hq][3] maximum, sum, correction
  float* acc = st + hq * 3;              // [hq][dim]
  T* cache = static_cast<T*>(br.cache) + static_cast<int64_t>(g) * br.chunk * dim;
  const int P = (dim + 1) / 2;
  for (int i = threadIdx.x; i < hq * P; i += kThreads) {
    const int h = i / P, p = i % P, d = 2 * p;
    const float* src = ph.proj + br.col_q + (g * hq + h) * dim;
    const float* bias = br.b_q + (g * hq + h) * dim;
    const float u = ldg_f(src + d) + bias[d], v = d + 1 < dim ? ldg_f(src + d + 1) + bias[d + 1] : 0.0f;
    float2 o = make_float2(u, v);
    if (p < br.rot_pairs) {
      const float2 cs = br.table[static_cast<int64_t>(slot) * br.rot_pairs + p];
      o = make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
    }
    qs[h * dim + d] = o.x * br.scale;
    if (d + 1 < dim) qs[h * dim + d + 1] = o.y * br.scale;
  }
  for (int i = threadIdx.x; i < hq * dim; i += kThreads) acc[i] = 0.0f;
  for (int i = threadIdx.x; i < hq; i += kThreads) {
    st[i * 3] = -FLT_MAX;
    st[i * 3 + 1] = 0.0f;
  }
  for (int jb = j0; jb < j1; jb += KT) {
    const int nk = min(KT, j1 - jb);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * P; i += kThreads) {
      const int jj = i / P, p = i % P, d = 2 * p, j = jb + jj;
      float u, v = 0.0f;
      T* cr = cache + static_cast<int64_t>(j) * dim + d;
      if (j == slot) {
        const float* src = ph.proj + br.col_k + g * dim + d;
        const float* bias = br.b_k + g * dim + d;
        u = ldg_f(src) + bias[0];
        cr[0] = from_f<T>(u);
        if (d + 1 < dim) {
          v = ldg_f(src + 1) + bias[1];
          cr[1] = from_f<T>(v);
        }
      } else {
        u = to_f(cr[0]);
        if (d + 1 < dim) v = to_f(cr[1]);
      }
      float2 o = make_float2(u, v);
      if (p < br.rot_pairs) {
        const float2 cs = br.table[static_cast<int64_t>(j) * br.rot_pairs + p];
        o = make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
      }
      kr[jj * ldk + d] = u;
      kt[jj * ldk + d] = o.x;
      if (d + 1 < dim) {
        kr[jj * ldk + d + 1] = v;
        kt[jj * ldk + d + 1] = o.y;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < hq * 32; i += kThreads) {
      const int h = i >> 5, jj = i & 31;
      float s0 = 0.0f, s1 = 0.0f;
      if (jj < nk) {
        const float *q = qs + h * dim, *k = kt + jj * ldk;
        int d = 0;
        for (; d + 1 < dim; d += 2) {
          s0 = fmaf(q[d], k[d], s0);
          s1 = fmaf(q[d + 1], k[d + 1], s1);
        }
        if (d < dim) s0 = fmaf(q[d], k[d], s0);
      }
      sc[i] = jj < nk ? s0 + s1 : -FLT_MAX;
    }
    __syncthreads();
    for (int h = wid; h < hq; h += kWarps) {
      const float s = sc[h * 32 + lane];
      const float m = st[h * 3], mn = fmaxf(m, warp_max(s));
      const float p = lane < nk ? expf(s - mn) : 0.0f, c = expf(m - mn);
      const float l = st[h * 3 + 1] * c + warp_sum(p);
      __syncwarp();
      sc[h * 32 + lane] = p;
      if (lane == 0) {
        st[h * 3] = mn;
        st[h * 3 + 1] = l;
        st[h * 3 + 2] = c;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < hq * dim; i += kThreads) {
      const int h = i / dim, d = i % dim;
      float t = acc[i] * st[h * 3 + 2];
      for (int jj = 0; jj < nk; ++jj) t = fmaf(sc[h * 32 + jj], kr[jj * ldk + d], t);
      acc[i] = t;
    }
  }
  __syncthreads();
  const int PS = dim + kAttnStats;
  for (int i = threadIdx.x; i < hq * dim; i += kThreads) {
    const int h = i / dim, d = i % dim;
    br.part[(static_cast<int64_t>(g * hq + h) * kAttnSplits + sp) * PS + kAttnStats + d] = acc[i];
  }
  for (int i = threadIdx.x; i < hq; i += kThreads) {
    float* pp = br.part + (static_cast<int64_t>(g * hq + i) * kAttnSplits + sp) * PS;
    pp[0] = st[i * 3];
    pp[1] = st[i * 3 + 1];
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    const unsigned int prev = atomicAdd(&br.arrive[g], 1u);
    *s_flag = prev == static_cast<unsigned int>(n_act - 1);
    if (*s_flag) br.arrive[g] = 0u;   // next use is a grid barrier away
  }
  __syncthreads();
  if (*s_flag) {
    __threadfence();
    for (int i = threadIdx.x; i < hq * dim; i += kThreads) {
      const int h = i / dim, d = i % dim;
      const float* pp = br.part + static_cast<int64_t>(g * hq + h) * kAttnSplits * PS;
      float M = -FLT_MAX;
      for (int s2 = 0; s2 < n_act; ++s2) M = fmaxf(M, ldg_f(pp + s2 * PS));
      float l = 0.0f, o = 0.0f;
      for (int s2 = 0; s2 < n_act; ++s2) {
        const float w = expf(ldg_f(pp + s2 * PS) - M);
        l += ldg_f(pp + s2 * PS + 1) * w;
        o += ldg_f(pp + s2 * PS + kAttnStats + d) * w;
      }
      br.out[(g * hq + h) * dim + d] = o / l * sigmoid_f(ldg_f(ph.proj + br.col_g + g * hq + h));
    }
  }
}

// Sum over the eight warps of a per-lane value; every thread gets its lane's total.
__device__ __forceinline__ float column_sum(float v, float* red /* [8][32] */) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  __syncthreads();
  red[wid * 32 + lane] = v;
  __syncthreads();
  float t = 0.0f;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) t += red[i * 32 + lane];
  return t;
}

// 32 value columns of one lightning head: a lane per column, the key rows dealt to the warps.
__device__ void lightning_item(const TokenPhase& ph, const TokenBranch& br, int item, int pos, float* sm) {
  const int nb = (br.vdim + 31) / 32, h = item / nb, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int c = (item % nb) * 32 + lane, dim = br.dim;
  float *q = sm, *k = q + dim, *red = k + dim;
  __syncthreads();
  for (int d = threadIdx.x; d < dim; d += kThreads) {
    q[d] = silu_f(ldg_f(ph.proj + br.col_q + h * dim + d));
    k[d] = silu_f(ldg_f(ph.proj + br.col_k + h * dim + d));
  }
  const bool live = c < br.vdim;
  const float v = live ? silu_f(ldg_f(ph.proj + br.col_v + h * br.vdim + c)) : 0.0f;
  const float dec = br.decay[h];
  float* S = br.state + static_cast<int64_t>(h) * dim * br.vdim + c;
  __syncthreads();
  float o = 0.0f;
  if (live) {
#pragma unroll 8
    for (int r = wid; r < dim; r += kWarps) {
      const float s0 = pos > 0 ? ldg_f(S + static_cast<int64_t>(r) * br.vdim) : 0.0f;
      const float s1 = fmaf(dec, s0, k[r] * v);
      S[static_cast<int64_t>(r) * br.vdim] = s1;
      o = fmaf(s1, q[r], o);
    }
  }
  o = column_sum(o, red);
  if (wid == 0 && live) br.out[h * br.vdim + c] = o;
}

// This token's value of convolution channel (ring channel rc, stacked projection column col), activated.
__device__ __forceinline__ float conv_channel(const TokenPhase& ph, const TokenBranch& br, int pos, int col, const float* taps, int rc,
                                              int ring_ld, bool owner) {
  const float now = ldg_f(ph.proj + col);
  float y = 0.0f;
  for (int j = 0; j < br.taps - 1; ++j) {
    const int p = pos - (br.taps - 1) + j;
    if (p >= 0) y = fmaf(taps[j], ldg_f(br.ring + static_cast<int64_t>(p % br.taps) * ring_ld + rc), y);
  }
  // the slot being overwritten is taps positions old: nobody reads it for this token
  if (owner) br.ring[static_cast<int64_t>(pos % br.taps) * ring_ld + rc] = now;
  return silu_f(fmaf(taps[br.taps - 1], now, y));
}

// dot of a low-rank row with a staged fp32 vector (rank rounded up to 8, both zero-padded)
template <typename T>
__device__ __forceinline__ float short_dot(const T* row, const float* x, int n) {
  constexpr int N = Chunk<T>::kN, U = 4;   // chunks in flight
  float acc = 0.0f;
  for (int i = 0; i < n; i += U * N) {
    Chunk<T> c[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i + u * N < n) c[u].load(row + i + u * N);
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i + u * N < n) acc = c[u].dot(x + i + u * N, acc);
  }
  return acc;
}

// 32 value columns of one delta-rule head.
template <typename T>
__device__ void delta_item(const TokenPhase& ph, const TokenBranch& br, int item, int pos, float* sm, float* red8) {
  const int nb = (br.vdim + 31) / 32, h = item / nb, vb = item % nb, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int dim = br.dim, grp = h / (br.H / br.G), c = vb * 32 + lane;
  const int qk = br.G * dim, ring_ld = 2 * qk + br.H * br.vdim;
  const int ra = (br.rank_a + 7) & ~7, rg = (br.rank_g + 7) & ~7;
  float *a1 = sm, *g1 = a1 + ra, *q = g1 + rg, *k = q + dim, *g = k + dim, *red = g + dim, *vs = red + kWarps * 32;
  __syncthreads();
  for (int i = threadIdx.x; i < ra; i += kThreads) a1[i] = i < br.rank_a ? ldg_f(ph.proj + br.col_a1 + i) : 0.0f;
  for (int i = threadIdx.x; i < rg; i += kThreads) g1[i] = i < br.rank_g ? ldg_f(ph.proj + br.col_g1 + i) : 0.0f;
  const bool own_qk = h % (br.H / br.G) == 0 && vb == 0;
  float ss[2] = {0.0f, 0.0f};
  for (int d = threadIdx.x; d < dim; d += kThreads) {
    const int ch = grp * dim + d;
    const float y = conv_channel(ph, br, pos, br.col_q + ch, br.conv_q + static_cast<int64_t>(ch) * br.taps, ch, ring_ld, own_qk);
    const float z = conv_channel(ph, br, pos, br.col_k + ch, br.conv_k + static_cast<int64_t>(ch) * br.taps, qk + ch, ring_ld, own_qk);
    q[d] = y;
    k[d] = z;
    ss[0] += y * y;
    ss[1] += z * z;
  }
  if (wid == kWarps - 1) {
    const int ch = h * br.vdim + c;
    vs[lane] = c < br.vdim ? conv_channel(ph, br, pos, br.col_v + ch, br.conv_v + static_cast<int64_t>(ch) * br.taps, 2 * qk + ch, ring_ld, true)
                           : 0.0f;
  }
  block_sum<2>(ss, red8);   // its barriers also publish a1, g1, q, k, vs
  const float sq = rsqrtf(ss[0] + 1e-6f) * rsqrtf(static_cast<float>(dim)), sk = rsqrtf(ss[1] + 1e-6f);
  const float amp = -expf(br.a_log[h]);
  for (int d = threadIdx.x; d < dim; d += kThreads) {
    q[d] *= sq;
    k[d] *= sk;
    const int ch = h * dim + d;
    const float z = short_dot(static_cast<const T*>(br.w_a2) + static_cast<int64_t>(ch) * ra, a1, ra) + br.dt_bias[ch];
    g[d] = expf(amp * softplus_f(z));
  }
  if (wid == kWarps - 1 && c < br.vdim) {
    const int ch = h * br.vdim + c;
    br.gate[ch] = short_dot(static_cast<const T*>(br.w_g2) + static_cast<int64_t>(ch) * rg, g1, rg);
  }
  const bool live = c < br.vdim;
  const float beta = sigmoid_f(ldg_f(ph.proj + br.col_b + h));
  float* S = br.state + static_cast<int64_t>(h) * dim * br.vdim + c;
  float s[32];   // dim <= 256: rows wid, wid + 8, ...
#pragma unroll
  for (int i = 0; i < 32; ++i) {
    const int r = wid + kWarps * i;
    s[i] = (r < dim && live && pos > 0) ? ldg_f(S + static_cast<int64_t>(r) * br.vdim) : 0.0f;
  }
  __syncthreads();
  float p = 0.0f;
#pragma unroll
  for (int i = 0; i < 32; ++i) {
    const int r = wid + kWarps * i;
    if (r < dim) {
      s[i] *= g[r];
      p = fmaf(s[i], k[r], p);
    }
  }
  const float u = beta * (vs[lane] - column_sum(p, red));
  float o = 0.0f;
#pragma unroll
  for (int i = 0; i < 32; ++i) {
    const int r = wid + kWarps * i;
    if (r < dim) {
      s[i] = fmaf(k[r], u, s[i]);
      if (live) S[static_cast<int64_t>(r) * br.vdim] = s[i];
      o = fmaf(s[i], q[r], o);
    }
  }
  o = column_sum(o, red);
  if (wid == 0 && live) br.out[h * br.vdim + c] = o;
}

// ---- parallel arrangement ----
// One CTA per SM with twice the threads: what a phase stages is staged once per SM.

// Experts of the token, chosen by every CTA for itself.
struct Routed {
  int32_t index[32];
  float weight[32];
};

// Items 0 .. n - 1 dealt to the threads, U loads of a thread in flight: put(i, load(i)).
template <int U, typename Load, typename Put>
__device__ __forceinline__ void batched(int n, int first, int threads, Load load, Put put) {
  for (int i0 = first; i0 < n; i0 += U * threads) {
    decltype(load(0)) v[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i0 + u * threads < n) v[u] = load(i0 + u * threads);
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i0 + u * threads < n) put(i0 + u * threads, v[u]);
  }
}
struct Pair4 {
  float4 a, b;
};
__device__ __forceinline__ float4 ldg4(const float* p) { return __ldcg(reinterpret_cast<const float4*>(p)); }
__device__ __forceinline__ float sq4(const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// V neighbouring columns.
template <int V>
struct Cols {
  float v[V];
  __device__ __forceinline__ void load(const float* p) {   // of memory that other CTAs write
    if constexpr (V == 4) {
      const float4 f = ldg4(p);
      v[0] = f.x;
      v[1] = f.y;
      v[2] = f.z;
      v[3] = f.w;
    } else {
      v[0] = ldg_f(p);
    }
  }
  template <typename U>
  __device__ __forceinline__ void get(const U* p) {   // weights, shared memory
    if constexpr (V == 4) {
      const float4 f = load4(p);
      v[0] = f.x;
      v[1] = f.y;
      v[2] = f.z;
      v[3] = f.w;
    } else {
      v[0] = to_f(*p);
    }
  }
  __device__ __forceinline__ void put(float* p) const {
    if constexpr (V == 4) store4(p, make_float4(v[0], v[1], v[2], v[3]));
    else *p = v[0];
  }
};

// The staged rows of ShiftNormArgs for one token. A thread keeps to its own columns, which lie in one group
// per turn; everything that does not depend on the norm is requested before it.
template <typename T, int V>
__device__ __forceinline__ void stage_shift_norm(const TokenArgs& a, const TokenPhase& ph, int64_t tok, int pos) {
  extern __shared__ __align__(16) float sm[];
  constexpr int U = V == 4 ? 1 : 2;   // turns in flight
  const TokenShift& f = ph.shift;
  const int W = a.width, gs = W / f.groups, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int g0 = wid / f.wpg, gstep = kListWarps / f.wpg, wj = wid % f.wpg, step = 32 * V * f.wpg;
  const bool active = g0 < gstep, writer = blockIdx.x == 0, shifted = f.shift != nullptr;
  const T* e = ph.first_token ? static_cast<const T*>(a.embed) + tok * a.ld_embed : nullptr;
  float *xs = sm, *part = sm + f.red;
  const float* prev = shifted ? f.state + ((pos + 1) & 1) * 2 * W : nullptr;
  float* next = shifted ? f.state + (pos & 1) * 2 * W : nullptr;
  for (int g = g0; active && g < f.groups; g += gstep) {
    float ss = 0.0f;
    const int end = (g + 1) * gs;
    for (int c0 = g * gs + (wj * 32 + lane) * V; c0 < end; c0 += U * step) {
      Cols<V> x[U], y1[U], z1[U], b1[U], y2[U], z2[U], b2[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * step;
        if (c >= end) break;
        if (e != nullptr) {
          x[u].get(e + c);
          continue;
        }
        x[u].load(f.x + c);
        y1[u].load(f.y1 + c);
        z1[u].load(f.z1 + c);
        b1[u].get(f.b1 + c);
        if (f.y2 != nullptr) {
          y2[u].load(f.y2 + c);
          z2[u].load(f.z2 + c);
          b2[u].get(f.b2 + c);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * step;
        if (c >= end) break;
#pragma unroll
        for (int k = 0; k < V; ++k) {
          if (e != nullptr) {
            x[u].v[k] *= a.embed_scale;
          } else {
            float r = y1[u].v[k] * sigmoid_f(z1[u].v[k] + b1[u].v[k]);
            if (f.y2 != nullptr) r += y2[u].v[k] * sigmoid_f(z2[u].v[k] + b2[u].v[k]);
            x[u].v[k] += r;
          }
          ss += x[u].v[k] * x[u].v[k];
        }
        x[u].put(xs + c);
        if (writer && f.x_out != nullptr) x[u].put(f.x_out + c);
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) part[g * f.wpg + wj] = ss;
  }
  // the first turns' weights and previous row are on their way over the barrier
  Cols<V> w0[U], s0[U], p0[U];
  auto request = [&](int c0, int end) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * step;
      if (c >= end) break;
      w0[u].get(f.w + c);
      if (!shifted) continue;
      s0[u].get(f.shift + c);
      if (pos > 0) p0[u].load(prev + c);
    }
  };
  if (active && g0 < f.groups) request(g0 * gs + (wj * 32 + lane) * V, (g0 + 1) * gs);
  __syncthreads();
  for (int g = g0; active && g < f.groups; g += gstep) {
    float ss = 0.0f;
    for (int k = 0; k < f.wpg; ++k) ss += part[g * f.wpg + k];
    const float sc = rsqrtf(ss / static_cast<float>(gs) + a.eps);
    const int begin = g * gs + (wj * 32 + lane) * V, end = (g + 1) * gs;
    for (int c0 = begin; c0 < end; c0 += U * step) {
      if (g != g0 || c0 != begin) request(c0, end);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * step;
        if (c >= end) break;
        Cols<V> h, m, mu[kTokenMixes], pm;
        if (f.n_mix > 0) {
          if (pos > 0) pm.load(prev + W + c);
#pragma unroll
          for (int i = 0; i < kTokenMixes; ++i) mu[i].get(f.mu[i] + c);
        }
        h.get(xs + c);
#pragma unroll
        for (int k = 0; k < V; ++k) h.v[k] *= sc * w0[u].v[k];
        h.put(xs + c);
        if (!shifted) continue;
#pragma unroll
        for (int k = 0; k < V; ++k) m.v[k] = fmaf((pos > 0 ? p0[u].v[k] : 0.0f) - h.v[k], s0[u].v[k], h.v[k]);
        m.put(sm + f.ld + c);
        if (writer) {
          h.put(f.h_out + c);
          h.put(next + c);
          if (f.n_mix > 0) m.put(next + W + c);
        }
        if (f.n_mix == 0) continue;
#pragma unroll
        for (int i = 0; i < kTokenMixes; ++i) {
          Cols<V> o;
#pragma unroll
          for (int k = 0; k < V; ++k) o.v[k] = fmaf((pos > 0 ? pm.v[k] : 0.0f) - m.v[k], mu[i].v[k], m.v[k]);
          o.put(sm + (2 + i) * f.ld + c);
        }
      }
    }
  }
  const int rows = shifted ? 2 + f.n_mix : 1, pad = f.ld - W;
  for (int i = threadIdx.x; i < rows * pad; i += kListThreads) sm[i / pad * f.ld + W + i % pad] = 0.0f;
  __syncthreads();
}

template <typename T>
__device__ __noinline__ void stage_list(const TokenArgs& a, const TokenPhase& ph, int64_t tok, int pos, float* red, Routed& routed) {
  extern __shared__ __align__(16) float sm[];
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  for (int i = 0; i < ph.n_ops; ++i) {
    const StageOp& op = ph.op[i];
    float* xs = sm + op.at;
    if (op.kind == kOpShiftNorm) {
      if (ph.shift.vec) stage_shift_norm<T, 4>(a, ph, tok, pos);
      else stage_shift_norm<T, 1>(a, ph, tok, pos);
    } else if (op.kind == kOpRmsNorm) {
      // every warp that takes part forms the sum by itself and stores its share: no barrier
      const int n4 = op.n >> 2, w0 = ph.route_top > 0 ? 1 : 0, parts = kListWarps - w0;
      if (wid >= w0) {
        constexpr int U = 8;   // 1024 columns at once
        float ss = 0.0f;
        for (int c = (op.n & ~3) + lane; c < op.n; c += 32) {
          const float v = ldg_f(op.src + c);
          ss += v * v;
        }
        for (int c0 = lane; c0 < n4; c0 += 32 * U) {
          float4 v[U];
#pragma unroll
          for (int u = 0; u < U; ++u) v[u] = c0 + 32 * u < n4 ? ldg4(op.src + 4 * (c0 + 32 * u)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int u = 0; u < U; ++u) ss += sq4(v[u]);
        }
        const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(op.n) + a.eps);
        for (int c = (wid - w0) * 32 + lane; c < n4; c += 32 * parts) {
          const float4 v = ldg4(op.src + 4 * c), w = load4(op.w + 4 * c);
          store4(xs + 4 * c, make_float4(v.x * sc * w.x, v.y * sc * w.y, v.z * sc * w.z, v.w * sc * w.w));
        }
        if (wid == w0)
          for (int c = (op.n & ~3) + lane; c < op.ld; c += 32) xs[c] = c < op.n ? ldg_f(op.src + c) * sc * op.w[c] : 0.0f;
      }
    } else if (op.kind == kOpCopy) {
      batched<1>(op.n >> 2, threadIdx.x, kListThreads, [&](int c) { return ldg4(op.src + 4 * c); }, [&](int c, const float4& v) { store4(xs + 4 * c, v); });
      for (int c = (op.n & ~3) + threadIdx.x; c < op.ld; c += kListThreads) xs[c] = c < op.n ? ldg_f(op.src + c) : 0.0f;
    } else if (op.kind == kOpRoute) {
      // one warp chooses (logits and scratch behind the copy), the others copy src2 to `at`
      float* z = xs + op.ld;
      if (wid == 0) {
        for (int c = lane; c < op.n; c += 32) z[c] = ldg_f(op.src + c);
        __syncwarp();
        route_token(z, op.w, op.n, ph.route_groups, ph.route_keep, ph.route_top, z + op.n, routed.index, routed.weight);
      } else {
        const int W = a.width, t = threadIdx.x - 32, threads = kListThreads - 32;
        batched<2>(W >> 2, t, threads, [&](int c) { return ldg4(op.src2 + 4 * c); }, [&](int c, const float4& v) { store4(xs + 4 * c, v); });
        for (int c = (W & ~3) + t; c < op.ld; c += threads) xs[c] = c < W ? ldg_f(op.src2 + c) : 0.0f;
      }
    } else if (op.kind == kOpGelu) {
      batched<1>(op.n >> 2, threadIdx.x, kListThreads, [&](int c) { return Pair4{ldg4(op.src + 4 * c), ldg4(op.src + op.ld + 4 * c)}; },
                 [&](int c, const Pair4& v) {
                   store4(xs + 4 * c, make_float4(gelu_tanh_f(v.a.x) * v.b.x, gelu_tanh_f(v.a.y) * v.b.y, gelu_tanh_f(v.a.z) * v.b.z,
                                                  gelu_tanh_f(v.a.w) * v.b.w));
                 });
    } else if (op.kind == kOpShared) {
      const float g = sigmoid_f(ldg_f(op.src2));
      batched<1>(op.n >> 2, threadIdx.x, kListThreads, [&](int c) { return Pair4{ldg4(op.src + 4 * c), ldg4(op.src + op.ld + 4 * c)}; },
                 [&](int c, const Pair4& v) {
                   store4(xs + 4 * c, make_float4(g * silu_f(v.a.x) * v.b.x, g * silu_f(v.a.y) * v.b.y, g * silu_f(v.a.z) * v.b.z,
                                                  g * silu_f(v.a.w) * v.b.w));
                 });
    } else if (op.kind == kOpExperts) {
      const int n4 = op.n >> 2;   // ld: number of experts; an identity output's columns are not read
      batched<2>(ph.route_top * n4, threadIdx.x, kListThreads,
                 [&](int c) {
                   const float* g = op.src + 8 * (c / n4) * n4 + 4 * (c % n4);
                   return Pair4{ldg4(g), ldg4(g + 4 * n4)};
                 },
                 [&](int c, const Pair4& v) {
                   const float w = routed.index[c / n4] < op.ld ? routed.weight[c / n4] : 0.0f;
                   store4(xs + 4 * c, make_float4(w * silu_f(v.a.x) * v.b.x, w * silu_f(v.a.y) * v.b.y, w * silu_f(v.a.z) * v.b.z,
                                                  w * silu_f(v.a.w) * v.b.w));
                 });
    } else if (op.kind == kOpHeadNorm) {
      const TokenBranch& br = ph.br[0];
      auto heads = [&](auto per_lane, auto at_once) {   // dim <= 32 per_lane; at_once heads in flight
        constexpr int E = decltype(per_lane)::value, B = decltype(at_once)::value;
        for (int h0 = wid; h0 < br.H; h0 += B * kListWarps) {
          float o[B][E], x[B][E], w[B][E];
#pragma unroll
          for (int j = 0; j < B; ++j)
#pragma unroll
            for (int u = 0; u < E; ++u) {
              const int h = h0 + j * kListWarps, d = lane + 32 * u, c = h * br.dim + d;
              const bool in = h < br.H && d < br.dim;
              o[j][u] = in ? ldg_f(op.src + c) : 0.0f;
              x[j][u] = in ? ldg_f(op.src2 + c) : 0.0f;
              w[j][u] = in ? op.w[c] : 0.0f;
            }
#pragma unroll
          for (int j = 0; j < B; ++j) {
            float ss = 0.0f;
#pragma unroll
            for (int u = 0; u < E; ++u) ss += o[j][u] * o[j][u];
            const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(br.dim) + a.eps);
            const int h = h0 + j * kListWarps;
#pragma unroll
            for (int u = 0; u < E; ++u)
              if (h < br.H && lane + 32 * u < br.dim) xs[h * br.dim + lane + 32 * u] = o[j][u] * sc * w[j][u] * silu_f(x[j][u]);
          }
        }
      };
      if (br.dim <= 64) heads(std::integral_constant<int, 2>(), std::integral_constant<int, 2>());
      else heads(std::integral_constant<int, 8>(), std::integral_constant<int, 1>());   // dim <= 256
      for (int c = op.n + threadIdx.x; c < op.ld; c += kListThreads) xs[c] = 0.0f;
    } else if (blockIdx.x == gridDim.x - 1 && wid == kListWarps - 1) {   // kOpLatentStore
      const TokenBranch& br = ph.br[0];
      const float* x = ph.proj + br.col_k;
      T* row = static_cast<T*>(br.cache) + static_cast<int64_t>(pos) * br.ld_cache;
      float ss = 0.0f;
#pragma unroll 8
      for (int c = lane; c < br.kv_rank; c += 32) {
        const float v = ldg_f(x + c);
        ss += v * v;
      }
      const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(br.kv_rank) + a.eps);
      batched<8>(br.kv_rank, lane, 32, [&](int c) { return ldg_f(x + c) * br.kv_norm[c]; }, [&](int c, float v) { row[c] = from_f<T>(v * sc); });
      const int half = br.rot_dim / 2;
      for (int p = lane; p < half; p += 32) {
        const float c0 = ldg_f(x + br.kv_rank + p), c1 = ldg_f(x + br.kv_rank + half + p);
        const float2 cs = br.table[static_cast<int64_t>(pos) * half + p];
        row[br.rot_col + p] = from_f<T>(c0 * cs.x - c1 * cs.y);
        row[br.rot_col + half + p] = from_f<T>(c1 * cs.x + c0 * cs.y);
      }
    }
  }
  __syncthreads();
}

// Row r of a product, this warp's part of it (all lanes get the sum).
template <typename T>
__device__ __forceinline__ float gemv_row(const TokenGemv& g, int r, const float* sm, int part, int wpr, const Routed& routed) {
  const T* W = static_cast<const T*>(g.W);
  if (g.mode == kGemvPlain) return row_dot<T>(W + static_cast<int64_t>(r) * g.K, sm + g.in, g.K, part, wpr);
  if (g.mode == kGemvExpertUp) {
    const int e = routed.index[r / g.per];
    if (e >= g.experts) return 0.0f;
    return row_dot<T>(W + (static_cast<int64_t>(e) * g.pitch + r % g.per) * g.K, sm + g.in, g.K, part, wpr);
  }
  float v = 0.0f;
  for (int k = 0; k < g.top; ++k) {
    const int e = routed.index[k];
    if (e < g.experts) v += row_part<T>(W + (static_cast<int64_t>(e) * g.pitch + r) * g.K, sm + g.in + k * g.K, g.K, part, wpr);
  }
  if (g.W2 != nullptr) v += row_part<T>(static_cast<const T*>(g.W2) + static_cast<int64_t>(r) * g.K2, sm + g.in2, g.K2, part, wpr);
  v = warp_sum(v);
  if (part == 0)
    for (int k = 0; k < g.top; ++k)
      if (routed.index[k] >= g.experts) v = fmaf(routed.weight[k], ldg_f(g.h + r), v);
  return v;
}

// 32 value columns of one wkv head (as delta_item: a lane per column, key rows dealt to the warps).
template <typename T>
__device__ __forceinline__ void wkv_item(const TokenPhase& ph, const TokenBranch& br, int item, int pos) {
  extern __shared__ __align__(16) float sm[];
  const int nb = (br.dim + 31) / 32, h = item / nb, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int dim = br.dim, c = (item % nb) * 32 + lane, rw = (br.rank_w + 7) & ~7;
  float *low = sm, *q = low + rw, *k = q + dim, *g = k + dim, *b = g + dim, *red = b + dim;
  const bool live = c < dim;
  float* S = br.state + static_cast<int64_t>(h) * dim * dim + c;
  float s[16];   // dim <= 256: rows wid, wid + 16, ...
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    const int r = wid + kListWarps * i;
    if (kListWarps * i >= dim) break;
    s[i] = (r < dim && live && pos > 0) ? ldg_f(S + static_cast<int64_t>(r) * dim) : 0.0f;
  }
  const float v = live ? ldg_f(ph.proj + br.col_v + h * dim + c) : 0.0f;
  __syncthreads();
  for (int i = threadIdx.x; i < rw; i += kListThreads) low[i] = i < br.rank_w ? tanhf(ldg_f(ph.proj + br.col_w1 + i)) : 0.0f;
  for (int d = threadIdx.x; d < dim; d += kListThreads) {
    const int ch = h * dim + d;
    q[d] = ldg_f(ph.proj + br.col_r + ch);
    k[d] = ldg_f(ph.proj + br.col_k + ch);
    b[d] = br.bonus[ch];
  }
  __syncthreads();
  for (int d = threadIdx.x; d < dim; d += kListThreads) {
    const int ch = h * dim + d;
    g[d] = expf(-expf(short_dot(static_cast<const T*>(br.w_w2) + static_cast<int64_t>(ch) * rw, low, rw) + br.w0[ch]));
  }
  __syncthreads();
  float o = 0.0f;
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    const int r = wid + kListWarps * i;
    if (kListWarps * i >= dim) break;
    if (r >= dim) continue;
    const float kv = k[r] * v;
    o = fmaf(fmaf(b[r], kv, s[i]), q[r], o);
    if (live) S[static_cast<int64_t>(r) * dim] = fmaf(g[r], s[i], kv);
  }
  __syncthreads();
  red[wid * 32 + lane] = o;
  __syncthreads();
  if (wid != 0 || !live) return;
  o = 0.0f;
#pragma unroll
  for (int i = 0; i < kListWarps; ++i) o += red[i * 32 + lane];
  br.out[h * dim + c] = o;
}

constexpr int kKeyGroups = kListThreads / 16;
template <typename T>
constexpr int kKeyCols = 16 * Chunk<T>::kN;   // latent columns of a key item

// Queries against the cache rows: W_uk^T q for one block of latent columns of a head; the first block also
// turns the rotated part. Threads: 16 column groups of one 16-byte chunk, kKeyGroups groups of key dimensions.
template <typename T>
__device__ __forceinline__ void latent_keys_item(const TokenBranch& br, int item, int pos) {
  extern __shared__ __align__(16) float sm[];
  constexpr int N = Chunk<T>::kN, COLS = kKeyCols<T>;
  const int nb = (br.rot_col + COLS - 1) / COLS, h = item / nb, r0 = item % nb * COLS;
  const int cg = threadIdx.x & 15, dg = threadIdx.x >> 4, col = r0 + cg * N;
  const float* q = br.q_up + h * (br.dim + br.rot_dim);
  float acc[N];
#pragma unroll
  for (int e = 0; e < N; ++e) acc[e] = 0.0f;
  if (col < br.ld_ukv) {
    const T* w = static_cast<const T*>(br.w_ukv) + static_cast<int64_t>(h) * br.dim * br.ld_ukv + col;
#pragma unroll 4
    for (int d = dg; d < br.dim; d += kKeyGroups) {
      Chunk<T> c;
      c.load(w + static_cast<int64_t>(d) * br.ld_ukv);
      const float x = ldg_f(q + d);
      float f[N];
      c.unpack(f);
#pragma unroll
      for (int e = 0; e < N; ++e) acc[e] = fmaf(x, f[e], acc[e]);
    }
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < N; ++e) sm[dg * (COLS + 1) + cg * N + e] = acc[e];
  __syncthreads();
  // fp32, or for bfloat16 caches high and low parts, one plane [H][ld_cache] after the other
  auto put = [&](int c, float v) {
    const int64_t i = static_cast<int64_t>(h) * br.ld_cache + c;
    if constexpr (sizeof(T) == 4) {
      static_cast<float*>(br.q_abs)[i] = v;
    } else {
      const T hi = from_f<T>(v);
      T* q2 = static_cast<T*>(br.q_abs);
      q2[i] = hi;
      q2[static_cast<int64_t>(br.H) * br.ld_cache + i] = from_f<T>(v - to_f(hi));
    }
  };
  for (int c = threadIdx.x; c < COLS; c += kListThreads) {
    float v = 0.0f;
#pragma unroll
    for (int g = 0; g < kKeyGroups; ++g) v += sm[g * (COLS + 1) + c];
    if (r0 + c < br.kv_rank) put(r0 + c, v * br.scale);
  }
  if (r0 == 0) {
    const int half = br.rot_dim / 2;
    for (int p = threadIdx.x; p < half; p += kListThreads) {
      const float u = ldg_f(q + br.dim + p), v = ldg_f(q + br.dim + half + p);
      const float2 cs = br.table[static_cast<int64_t>(pos) * half + p];
      put(br.rot_col + p, (u * cs.x - v * cs.y) * br.scale);
      put(br.rot_col + half + p, (v * cs.x + u * cs.y) * br.scale);
    }
  }
}

// Position ranges in use for L cached positions, and their length (whole tiles).
__device__ __forceinline__ int latent_ranges(int L, int splits, int& per) {
  const int tiles = (L + kLatentKeys - 1) / kLatentKeys, each = (tiles + splits - 1) / splits;
  per = each * kLatentKeys;
  return (tiles + each - 1) / each;
}

// kLatentHeadsF32 query heads over one range of cached positions: running maximum, sum and the weighted sum
// of the latents per head. Scores: a warp per head, a lane per position. Sums: a thread per pair of columns.
__device__ __forceinline__ void latent_scan_f32_item(const TokenBranch& br, int item, int pos) {
  extern __shared__ __align__(16) float sm[];
  using T = float;
  constexpr int N = Chunk<T>::kN, HB = kLatentHeadsF32, KT = kLatentKeys;
  const int blk = item / br.splits, sp = item % br.splits;
  int per;
  const int n_act = latent_ranges(pos + 1, br.splits, per);
  if (sp >= n_act) return;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, ldc = br.ld_cache;
  const int j0 = sp * per, j1 = min(pos + 1, j0 + per);
  const int chunks = ldc / N, pitch = chunks | 1;       // 16-byte chunks per row; odd pitch: conflict-free
  float* qs = sm;                                       // [HB][ldc]
  float* ps = qs + HB * ldc;                            // [HB][KT] scores, then weights
  float* st = ps + HB * KT;                             // [HB] correction of the sums
  uint4* tiles = reinterpret_cast<uint4*>(st + HB);     // [br.buffers][KT][pitch]
  const uint4* cache = reinterpret_cast<const uint4*>(static_cast<const T*>(br.cache));
  auto request = [&](int jb) {   // rows past the range stay what they were: their weights are zero
    uint4* tile = tiles + ((jb - j0) / KT & (br.buffers - 1)) * KT * pitch;
    const int n = min(KT, j1 - jb) * chunks;
#pragma unroll 2
    for (int i = threadIdx.x; i < n; i += kListThreads) cp_async16(tile + i / chunks * pitch + i % chunks, cache + static_cast<int64_t>(jb) * chunks + i);
    cp_async_commit();
  };
  request(j0);
  {
    const int c4 = ldc >> 2, valid = (min(br.H, (blk + 1) * HB) - blk * HB) * c4;
    const float* src = static_cast<const float*>(br.q_abs) + static_cast<int64_t>(blk) * HB * ldc;
    batched<2>(HB * c4, threadIdx.x, kListThreads, [&](int i) { return i < valid ? ldg4(src + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f); },
               [&](int i, const float4& x) { store4(qs + 4 * i, x); });
  }
  float m = -FLT_MAX, l = 0.0f;   // of head wid (the first HB warps)
  float2 acc[HB];   // kv_rank <= 2 kListThreads
#pragma unroll
  for (int h = 0; h < HB; ++h) acc[h] = make_float2(0.0f, 0.0f);
  const int col = 2 * threadIdx.x;
  for (int jb = j0; jb < j1; jb += KT) {
    const int nk = min(KT, j1 - jb);
    const uint4* tile = tiles + ((jb - j0) / KT & (br.buffers - 1)) * KT * pitch;
    const bool ahead = br.buffers > 1 && jb + KT < j1;
    if (ahead) request(jb + KT);
    if (ahead) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();
    if (wid < HB) {
      const float* q = qs + wid * ldc;
      float s0 = 0.0f, s1 = 0.0f;
#pragma unroll 2
      for (int c = 0; c < chunks; ++c) {
        Chunk<T> k;
        k.w = *reinterpret_cast<const decltype(k.w)*>(tile + lane * pitch + c);
        if (c & 1) s1 = k.dot(q + c * N, s1);
        else s0 = k.dot(q + c * N, s0);
      }
      const float s = lane < nk ? s0 + s1 : -FLT_MAX;
      const float mn = fmaxf(m, warp_max(s));
      const float p = lane < nk ? expf(s - mn) : 0.0f, c = expf(m - mn);
      l = l * c + warp_sum(p);
      m = mn;
      ps[wid * KT + lane] = p;
      if (lane == 0) st[wid] = c;
    }
    __syncthreads();
    if (col < br.kv_rank) {
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        acc[h].x *= st[h];
        acc[h].y *= st[h];
      }
      const T* row = reinterpret_cast<const T*>(tile) + col;
#pragma unroll 1
      for (int j = 0; j < nk; j += 4) {
        float x[4], y[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const bool in = j + u < nk;   // what lies behind the range need not be a number
          x[u] = in ? to_f(row[(j + u) * pitch * N]) : 0.0f;
          y[u] = in ? to_f(row[(j + u) * pitch * N + 1]) : 0.0f;
        }
#pragma unroll
        for (int h = 0; h < HB; ++h) {
          const float4 w = *reinterpret_cast<const float4*>(ps + h * KT + j);
          acc[h].x = fmaf(w.x, x[0], fmaf(w.y, x[1], fmaf(w.z, x[2], fmaf(w.w, x[3], acc[h].x))));
          acc[h].y = fmaf(w.x, y[0], fmaf(w.y, y[1], fmaf(w.z, y[2], fmaf(w.w, y[3], acc[h].y))));
        }
      }
    }
    __syncthreads();   // before this tile's place or the weights are written again
    if (br.buffers == 1 && jb + KT < j1) request(jb + KT);
  }
  const int PS = br.rot_col + kAttnStats4;
  auto part = [&](int h) { return br.part + (static_cast<int64_t>(blk * HB + h) * br.splits + sp) * PS; };
  if (col < br.kv_rank) {
#pragma unroll
    for (int h = 0; h < HB; ++h)   // rows end on an even column: rot_col is a multiple of eight
      if (blk * HB + h < br.H) *reinterpret_cast<float2*>(part(h) + kAttnStats4 + col) = acc[h];
  }
  if (lane == 0 && wid < HB && blk * HB + wid < br.H) {
    part(wid)[0] = m;
    part(wid)[1] = l;
  }
}

// The same for bfloat16 caches on the tensor cores: kLatentHeads heads are the rows of the products. Queries
// and weights are split into a bfloat16 sum of two terms (16 mantissa bits, fp32 sums). Scores: a warp per 16
// positions and eighth of the columns; sums: a warp per 32 NB columns.
template <int NB>
__device__ __forceinline__ void latent_scan_bf16_item(const TokenBranch& br, int item, int pos) {
  extern __shared__ __align__(16) float sm[];
  using bf16 = __nv_bfloat16;
  constexpr int HB = kLatentHeads, KT = kLatentKeys, LP = KT + 8;
  static_assert(HB == kListWarps, "a warp per head");
  const int blk = item / br.splits, sp = item % br.splits;
  int per;
  const int n_act = latent_ranges(pos + 1, br.splits, per);
  if (sp >= n_act) return;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, ldc = br.ld_cache, cols = (ldc + 15) & ~15, pitch = cols + 8;
  const int j0 = sp * per, j1 = min(pos + 1, j0 + per), chunks = ldc / 8;
  bf16* qh = reinterpret_cast<bf16*>(sm);               // [HB][pitch] queries, high and low
  bf16* ql = qh + HB * pitch;
  bf16* ph = ql + HB * pitch;                           // [HB][LP] weights, high and low
  bf16* pl = ph + HB * LP;
  float* sc = reinterpret_cast<float*>(pl + HB * LP);   // [8][HB][KT + 4] scores per eighth of the columns
  float* st = sc + 8 * HB * (KT + 4);                   // [HB] correction of the sums
  bf16* tiles = reinterpret_cast<bf16*>(st + HB);       // [br.buffers][KT][pitch]
  const bf16* cache = static_cast<const bf16*>(br.cache);
  auto tile_at = [&](int jb) { return tiles + ((jb - j0) / KT & (br.buffers - 1)) * KT * pitch; };
  auto request = [&](int jb) {   // a warp per row; rows past the end are zero
    bf16* tile = tile_at(jb);
    for (int r = wid; r < KT; r += kListWarps) {
      const bf16* src = cache + static_cast<int64_t>(jb + r) * ldc;
      for (int c = lane; c < chunks; c += 32) {
        if (jb + r < j1) cp_async16(tile + r * pitch + c * 8, src + c * 8);
        else *reinterpret_cast<uint4*>(tile + r * pitch + c * 8) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    cp_async_commit();
  };
  for (int r = wid; r < 2 * HB; r += kListWarps) {   // queries: a warp per row and plane
    const int h = blk * HB + r % HB;
    const bf16* src = static_cast<const bf16*>(br.q_abs) + (static_cast<int64_t>(r / HB) * br.H + h) * ldc;
    for (int c = lane; c < chunks; c += 32) {
      if (h < br.H) cp_async16(qh + r * pitch + c * 8, src + c * 8);
      else *reinterpret_cast<uint4*>(qh + r * pitch + c * 8) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
  request(j0);
  if (cols > ldc)   // columns up to the product's slice of 16
    for (int i = threadIdx.x; i < 2 * HB + br.buffers * KT; i += kListThreads)
      *reinterpret_cast<uint4*>((i < 2 * HB ? qh + i * pitch : tiles + (i - 2 * HB) * pitch) + ldc) = make_uint4(0u, 0u, 0u, 0u);
  const int slice = wid >> 1, n0 = (wid & 1) * 16, steps = cols / 16, s0 = steps * slice / 8, s1 = steps * (slice + 1) / 8;
  const int c0 = wid * NB * 32;   // the warp's columns of the sums
  float m = -FLT_MAX, l = 0.0f;   // of head wid
  float acc[NB * 4][4];
#pragma unroll
  for (int t = 0; t < NB * 4; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[t][e] = 0.0f;
  for (int jb = j0; jb < j1; jb += KT) {
    const int nk = min(KT, j1 - jb);
    const bf16* tile = tile_at(jb);
    const bool ahead = br.buffers > 1 && jb + KT < j1;
    if (ahead) request(jb + KT);
    if (ahead) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();
    {
      float s[2][4] = {};
#pragma unroll 2
      for (int k = s0; k < s1; ++k) {
        uint32_t Ah[4], Al[4], B[4];
        ldsm_a(Ah, qh, pitch, 0, k * 16, lane);
        ldsm_a(Al, ql, pitch, 0, k * 16, lane);
        ldsm_b(B, tile, pitch, k * 16, n0, lane);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma_bf16(s[t], Ah, B[2 * t], B[2 * t + 1]);
          mma_bf16(s[t], Al, B[2 * t], B[2 * t + 1]);
        }
      }
      float* dst = sc + (slice * HB + (lane >> 2)) * (KT + 4) + n0 + (lane & 3) * 2;
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int f = 0; f < 2; ++f)
          *reinterpret_cast<float2*>(dst + f * 8 * (KT + 4) + t * 8) = make_float2(s[t][2 * f], s[t][2 * f + 1]);
    }
    __syncthreads();
    {
      const float* src = sc + wid * (KT + 4) + lane;
      float s = 0.0f;
#pragma unroll
      for (int k = 0; k < 8; ++k) s += src[k * HB * (KT + 4)];
      if (lane >= nk) s = -FLT_MAX;
      const float mn = fmaxf(m, warp_max(s));
      const float p = lane < nk ? expf(s - mn) : 0.0f, c = expf(m - mn);
      l = l * c + warp_sum(p);
      m = mn;
      const bf16 hi = __float2bfloat16(p);
      ph[wid * LP + lane] = hi;
      pl[wid * LP + lane] = __float2bfloat16(p - __bfloat162float(hi));
      if (lane == 0) st[wid] = c;
    }
    __syncthreads();
    if (c0 < br.kv_rank) {
      const float f0 = st[lane >> 2], f1 = st[(lane >> 2) + 8];
#pragma unroll
      for (int t = 0; t < NB * 4; ++t) {
        acc[t][0] *= f0;
        acc[t][1] *= f0;
        acc[t][2] *= f1;
        acc[t][3] *= f1;
      }
#pragma unroll
      for (int k = 0; k < KT; k += 16) {
        uint32_t Ah[4], Al[4];
        ldsm_a(Ah, ph, LP, 0, k, lane);
        ldsm_a(Al, pl, LP, 0, k, lane);
#pragma unroll
        for (int t = 0; t < NB * 4; t += 2) {
          if (c0 + t * 8 >= br.kv_rank) break;
          uint32_t B[4];
          ldsm_b_trans(B, tile, pitch, k, c0 + t * 8, lane);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mma_bf16(acc[t + e], Ah, B[2 * e], B[2 * e + 1]);
            mma_bf16(acc[t + e], Al, B[2 * e], B[2 * e + 1]);
          }
        }
      }
    }
    __syncthreads();   // before this tile's place or the weights are written again
    if (br.buffers == 1 && jb + KT < j1) request(jb + KT);
  }
  const int PS = br.rot_col + kAttnStats4;
  auto part = [&](int h) { return br.part + (static_cast<int64_t>(blk * HB + h) * br.splits + sp) * PS; };
#pragma unroll
  for (int t = 0; t < NB * 4; ++t) {
    const int col = c0 + t * 8 + (lane & 3) * 2;
    if (col >= br.kv_rank) break;
#pragma unroll
    for (int f = 0; f < 2; ++f) {
      const int h = (lane >> 2) + 8 * f;
      if (blk * HB + h < br.H) *reinterpret_cast<float2*>(part(h) + kAttnStats4 + col) = make_float2(acc[t][2 * f], acc[t][2 * f + 1]);
    }
  }
  if (lane == 0 && blk * HB + wid < br.H) {
    part(wid)[0] = m;
    part(wid)[1] = l;
  }
}

constexpr int kOutParts = kLatentOutParts;

// kLatentOutRows value rows of a head: merges the head's ranges, then W_uv times the mean latent, gated.
template <typename T>
__device__ __forceinline__ void latent_out_item(const TokenPhase& ph, const TokenBranch& br, int item, int pos) {
  extern __shared__ __align__(16) float sm[];
  const int nb = (br.vdim + kLatentOutRows - 1) / kLatentOutRows, h = item / nb, r0 = item % nb * kLatentOutRows;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, PS = br.rot_col + kAttnStats4;
  int per;
  const int n_act = latent_ranges(pos + 1, br.splits, per);
  // [rot_col] mean latent, [splits] weights of the ranges, [kOutParts][rot_col] partial sums
  float *o = sm, *sums = o + br.rot_col, *w = sums + kOutParts * br.rot_col;
  // the weight rows are requested before the ranges are merged: ROWS rows per warp, HELD chunks per lane of each
  constexpr int N = Chunk<T>::kN, ROWS = kLatentOutRows / kListWarps, HELD = 2;
  const int ld = br.ld_ukv;
  const T* rows = static_cast<const T*>(br.w_ukv) + (static_cast<int64_t>(br.row_uv) + h * br.vdim) * ld;
  Chunk<T> held[ROWS][HELD];
#pragma unroll
  for (int u = 0; u < ROWS; ++u)
#pragma unroll
    for (int k = 0; k < HELD; ++k)
      if (r0 + wid + u * kListWarps < br.vdim && (k * 32 + lane) * N < ld)
        held[u][k].load(rows + static_cast<int64_t>(r0 + wid + u * kListWarps) * ld + (k * 32 + lane) * N);
  const float gate = sigmoid_f(ldg_f(ph.proj + br.col_g + h));
  const float* part = br.part + static_cast<int64_t>(h) * br.splits * PS;
  __syncthreads();
  if (wid == 0) {
    float m = -FLT_MAX;
    for (int s = lane; s < n_act; s += 32) m = fmaxf(m, ldg_f(part + static_cast<int64_t>(s) * PS));
    m = warp_max(m);
    float l = 0.0f;
    for (int s = lane; s < n_act; s += 32) {
      const float e = expf(ldg_f(part + static_cast<int64_t>(s) * PS) - m);
      w[s] = e;
      l += e * ldg_f(part + static_cast<int64_t>(s) * PS + 1);
    }
    l = 1.0f / warp_sum(l);
    __syncwarp();
    for (int s = lane; s < n_act; s += 32) w[s] *= l;
  }
  __syncthreads();
  {   // four columns per thread; the ranges are dealt to kOutParts groups of threads
    const int quads = br.rot_col / 4, n = quads * kOutParts;
    for (int i = threadIdx.x; i < n; i += kListThreads) {
      const int c = i % quads * 4, first = i / quads;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int s = first; s < n_act; s += kOutParts) {
        const float4 x = ldg4(part + static_cast<int64_t>(s) * PS + kAttnStats4 + c);
        v = make_float4(fmaf(w[s], x.x, v.x), fmaf(w[s], x.y, v.y), fmaf(w[s], x.z, v.z), fmaf(w[s], x.w, v.w));
      }
      store4(sums + first * br.rot_col + c, v);
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < br.rot_col; c += kListThreads) {
    float v = 0.0f;
#pragma unroll
    for (int g = 0; g < kOutParts; ++g) v += sums[g * br.rot_col + c];
    o[c] = c < br.kv_rank ? v : 0.0f;
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < ROWS; ++u) {
    float v = 0.0f;
#pragma unroll
    for (int k = 0; k < HELD; ++k)
      if ((k * 32 + lane) * N < ld) v = held[u][k].dot(o + (k * 32 + lane) * N, v);
    const int r = r0 + wid + u * kListWarps;
    for (int c = HELD * 32 + lane; c * N < ld && r < br.vdim; c += 32) {
      Chunk<T> w1;
      w1.load(rows + static_cast<int64_t>(r) * ld + c * N);
      v = w1.dot(o + c * N, v);
    }
    v = warp_sum(v);
    if (lane == 0 && r < br.vdim) br.out[h * br.vdim + r] = v * gate;
  }
}

template <typename T>
__device__ __forceinline__ void list_item(const TokenPhase& ph, int item, int pos) {
  const TokenBranch& br = ph.br[0];
  if (br.kind == kTokWkv) wkv_item<T>(ph, br, item, pos);
  else if (br.kind == kTokLatentKeys) latent_keys_item<T>(br, item, pos);
  else if (br.kind == kTokLatentOut) latent_out_item<T>(ph, br, item, pos);
  else if constexpr (sizeof(T) == 2) br.kv_rank <= 512 ? latent_scan_bf16_item<1>(br, item, pos) : latent_scan_bf16_item<2>(br, item, pos);
  else latent_scan_f32_item(br, item, pos);
}

// Staging, products, items. The items lie at the front of the grid, so rows start behind them.
template <typename T>
__device__ unsigned long long list_phase(const TokenArgs& a, const TokenPhase& ph, int64_t tok, int pos, float* sm, float* red, float* part_red,
                                         Routed& routed) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  if (ph.n_ops > 0) stage_list<T>(a, ph, tok, pos, red, routed);
  unsigned long long best = 0ull;
  int total = 0;
  for (int i = 0; i < ph.n_gemv; ++i) total += ph.gemv[i].rows;
  const int items = ph.n_branch > 0 ? ph.br[0].items : 0;
  int cta = static_cast<int>(blockIdx.x) - items % static_cast<int>(gridDim.x);
  if (cta < 0) cta += gridDim.x;
  const int wpr = ph.wpr, groups = kListWarps / (wpr > 0 ? wpr : 1), part = wpr > 0 ? wid % wpr : 0;
  auto find = [&](int n, int& r) {
    int i = 0;
    while (n >= ph.gemv[i].rows) n -= ph.gemv[i++].rows;
    r = n;
    return i;
  };
  auto finish = [&](const TokenGemv& g, int r, float v) {
    g.y[r] = v;
    if (ph.is_head) {
      const unsigned long long k = argmax_key(v, r);
      best = k > best ? k : best;
    }
  };
  if (wpr == 1) {
    for (int n = cta * kListWarps + wid; n < total; n += gridDim.x * kListWarps) {
      int r;
      const TokenGemv& g = ph.gemv[find(n, r)];
      const float v = gemv_row<T>(g, r, sm, 0, 1, routed);
      if (lane == 0) finish(g, r, v);
    }
  } else {
    for (int nb = cta * groups; nb < total; nb += gridDim.x * groups) {
      const int n = nb + wid / wpr;
      int r = 0;
      float v = 0.0f;
      const TokenGemv& g = ph.gemv[n < total ? find(n, r) : 0];
      if (n < total) v = gemv_row<T>(g, r, sm, part, wpr, routed);
      if (lane == 0) part_red[wid] = v;
      __syncthreads();
      if (part == 0 && lane == 0 && n < total) {
        float t = 0.0f;
        for (int w = 0; w < wpr; ++w) t += part_red[wid + w];
        finish(g, r, t);
      }
      __syncthreads();
    }
  }
  for (int it = blockIdx.x; it < items; it += gridDim.x) {
    __syncthreads();
    list_item<T>(ph, it, pos);
  }
  return best;
}

template <typename T, int kThreads>
__device__ void prefetch_phase(const TokenPhase& ph) {
  if (ph.extra != nullptr) {
    const char* base = static_cast<const char*>(ph.extra);
    for (int64_t i = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x; i < ph.extra_bytes / 128; i += static_cast<int64_t>(gridDim.x) * kThreads)
      prefetch_l2(base + i * 128);
  }
  for (int s = 0; s < ph.n_gemv; ++s) {
    const TokenGemv& g = ph.gemv[s];
    if (g.mode != kGemvPlain) continue;   // which experts is not known yet
    const char* base = static_cast<const char*>(g.W);
    const int64_t lines = static_cast<int64_t>(g.rows) * g.K * sizeof(T) / 128;
    for (int64_t i = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x; i < lines; i += static_cast<int64_t>(gridDim.x) * kThreads)
      prefetch_l2(base + i * 128);
  }
}

// LIST: every phase is a kStageList phase (parallel arrangement); otherwise none is.
template <typename T, bool LIST>
__global__ void __launch_bounds__(LIST ? kListThreads : kThreads, LIST ? 1 : 2) hybrid_token_kernel(const __grid_constant__ TokenArgs a) {
  constexpr int kThreads = token_threads(LIST), kWarps = kThreads / 32;
  extern __shared__ __align__(16) float sm[];
  __shared__ TokenPhase ph_s[2];
  __shared__ float red[2 * kWarps];
  __shared__ float part_red[kWarps];
  __shared__ unsigned long long best_s[kWarps];
  __shared__ int s_flag;
  __shared__ Routed routed;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  unsigned int epoch = 0;
  int pos = a.counters[0];
  int64_t tok = *a.cur_token;
  unsigned long long* words = reinterpret_cast<unsigned long long*>(a.sync + 128);
  bool alive = true;
  auto fetch = [&](int i) {   // phase descriptions are read one phase ahead
    const int* src = reinterpret_cast<const int*>(a.phases + i);
    int* dst = reinterpret_cast<int*>(&ph_s[i & 1]);
    for (int w = threadIdx.x; w < static_cast<int>(sizeof(TokenPhase) / 4); w += kThreads) dst[w] = src[w];
  };
  for (int t = 0; t < a.n_tokens && alive; ++t) {
    fetch(0);
    __syncthreads();
    for (int i = 0; i < a.n_phases; ++i) {
      const TokenPhase& ph = ph_s[i & 1];
      unsigned long long best = 0ull;
      if constexpr (LIST) {
        best = list_phase<T>(a, ph, tok, pos, sm, red, part_red, routed);
      } else if (ph.is_mix) {
        int first = 0;
        for (int b = 0; b < ph.n_branch; ++b) {
          const TokenBranch& br = ph.br[b];
          for (int it = blockIdx.x; it < first + br.items; it += gridDim.x) {
            if (it < first) continue;
            __syncthreads();
            if (br.kind == kTokAttention) attention_item<T>(ph, br, it - first, pos, sm, &s_flag);
            else if (br.kind == kTokLightning) lightning_item(ph, br, it - first, pos, sm);
            else delta_item<T>(ph, br, it - first, pos, sm, red);
          }
          first += br.items;
        }
      } else {
        if (ph.stage == kStageNorm) {
          stage_norm<T>(a, ph, tok, sm, red);
        } else if (ph.stage == kStageGlu) {
          for (int c = threadIdx.x; c < ph.ffp; c += kThreads) sm[c] = clamped_glu_f(ldg_f(ph.gu + c), ldg_f(ph.gu + ph.ffp + c), ph.limit);
          __syncthreads();
        } else {
          stage_mixed(a, ph, sm, red);
        }
        const int wpr = ph.wpr, groups = kWarps / wpr, part = wid % wpr;
        const int rows0 = ph.gemv[0].rows, total = rows0 + (ph.n_gemv > 1 ? ph.gemv[1].rows : 0);
        if (wpr == 1) {
          for (int n = blockIdx.x * kWarps + wid; n < total; n += gridDim.x * kWarps) {
            const TokenGemv& g = ph.gemv[n < rows0 ? 0 : 1];
            const int r = n < rows0 ? n : n - rows0;
            const float v = row_dot<T>(static_cast<const T*>(g.W) + static_cast<int64_t>(r) * g.K, sm + g.in, g.K, 0, 1);
            if (lane == 0) {
              g.y[r] = v;
              if (ph.is_head) {
                const unsigned long long k = argmax_key(v, r);
                best = k > best ? k : best;
              }
            }
          }
        } else {
          // wpr warps share a row; the block walks its rows in step
          for (int nb = blockIdx.x * groups; nb < total; nb += gridDim.x * groups) {
            const int n = nb + wid / wpr;
            float v = 0.0f;
            const TokenGemv& g = ph.gemv[n < rows0 ? 0 : 1];
            const int r = n < rows0 ? n : n - rows0;
            if (n < total) v = row_dot<T>(static_cast<const T*>(g.W) + static_cast<int64_t>(r) * g.K, sm + g.in, g.K, part, wpr);
            if (lane == 0) part_red[wid] = v;
            __syncthreads();
            if (part == 0 && lane == 0 && n < total) {
              float s = 0.0f;
              for (int w = 0; w < wpr; ++w) s += part_red[wid + w];
              g.y[r] = s;
              if (ph.is_head) {
                const unsigned long long k = argmax_key(s, r);
                best = k > best ? k : best;
              }
            }
            __syncthreads();
          }
        }
      }
      if (ph.is_head && a.out_tokens != nullptr) {
        if (lane == 0) best_s[wid] = best;
        __syncthreads();
        if (threadIdx.x == 0) {
#pragma unroll
          for (int w = 1; w < kWarps; ++w) best = best_s[w] > best ? best_s[w] : best;
          atomicMax(&words[t & 1], best);
        }
      }
      if (ph.prefetch >= 0) prefetch_phase<T, kThreads>(a.phases[ph.prefetch]);
      if (i + 1 < a.n_phases) fetch(i + 1);
      if (i + 1 == a.n_phases && a.out_tokens == nullptr) break;   // logits are complete at the end of the kernel
      if (!(alive = grid_barrier(a.sync, a.status, 91, epoch))) break;
    }
    if (!alive || a.out_tokens == nullptr) break;
    const unsigned long long wv = *reinterpret_cast<volatile unsigned long long*>(&words[t & 1]);
    tok = static_cast<int64_t>(0xFFFFFFFFu - static_cast<unsigned>(wv & 0xFFFFFFFFull));
    if (blockIdx.x == 0 && threadIdx.x == 0) {
      a.out_tokens[a.out_offset + t] = tok;
      words[(t + 1) & 1] = 0ull;   // last read one barrier ago
    }
    pos += 1;
  }
  if (blockIdx.x == 0 && threadIdx.x == 0 && a.out_tokens != nullptr) {
    a.counters[0] = pos;
    a.counters[1] += a.n_tokens;
    *a.cur_token = tok;
  }
}

}  // namespace

size_t token_smem_bytes(int stage_floats, const TokenPhase* phases, int n) {
  size_t need = static_cast<size_t>(stage_floats);
  for (int i = 0; i < n; ++i) {
    for (int b = 0; phases[i].is_mix && b < phases[i].n_branch; ++b) {
      const TokenBranch& br = phases[i].br[b];
      size_t f = 0;
      if (phases[i].stage == kStageList) continue;   // counted by the caller
      if (br.kind == kTokAttention) {
        const size_t hq = br.H / br.G, kt = br.dim <= 128 ? 32 : (br.dim <= 256 ? 16 : (br.dim <= 512 ? 8 : 4));
        f = 2 * hq * br.dim + 2 * kt * (br.dim + 1) + hq * 35;
      } else if (br.kind == kTokLightning) {
        f = 2 * br.dim + kWarps * 32;
      } else {
        f = br.rank_a + br.rank_g + 16 + 3 * br.dim + kWarps * 32 + 32;
      }
      if (f > need) need = f;
    }
  }
  return need * 4;
}

template <typename T>
int token_grid(size_t smem, bool list, int* grid) {
  auto* kernel = list ? hybrid_token_kernel<T, true> : hybrid_token_kernel<T, false>;
  int dev = 0, coop = 0, per_sm = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e == cudaSuccess) e = cudaDeviceGetAttribute(&coop, cudaDevAttrCooperativeLaunch, dev);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e == cudaSuccess) e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kernel, token_threads(list), smem);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "hybrid token kernel: %s", cudaGetErrorString(e));
  CTDK_REQUIRE(coop != 0 && per_sm >= 1, "hybrid token kernel: no cooperative launch with %zu bytes of shared memory", smem);
  const int most = list ? 1 : 2;   // CTAs per SM the kernel is made for
  *grid = sm_count() * (per_sm > most ? most : per_sm);
  return CTDK_OK;
}

template <typename T>
int launch_token_kernel(const TokenArgs& a, bool list, int grid, size_t smem, cudaStream_t s) {
  if (cudaMemsetAsync(a.sync, 0, a.sync_words * sizeof(unsigned int), s) != cudaSuccess)
    return fail(CTDK_ELAUNCH, "hybrid token kernel: clearing the barrier words failed");
  TokenArgs args = a;
  void* params[] = {&args};
  const cudaError_t e = cudaLaunchCooperativeKernel(list ? reinterpret_cast<const void*>(hybrid_token_kernel<T, true>) : reinterpret_cast<const void*>(hybrid_token_kernel<T, false>), dim3(grid), dim3(token_threads(list)),
                                                    params, smem, s);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "hybrid token kernel: %s", cudaGetErrorString(e));
  return check_launch("hybrid token kernel");
}

template int token_grid<float>(size_t, bool, int*);
template int token_grid<__nv_bfloat16>(size_t, bool, int*);
template int launch_token_kernel<float>(const TokenArgs&, bool, int, size_t, cudaStream_t);
template int launch_token_kernel<__nv_bfloat16>(const TokenArgs&, bool, int, size_t, cudaStream_t);

}  // namespace hybrid
}  // namespace ctdk
