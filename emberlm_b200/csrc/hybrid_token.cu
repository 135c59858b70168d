// Persistent token kernel of the layer-list family (hybrid_token.h). Per layer with two branches:
//   [sandwich norms + stacked input projection] | [mix: attention key ranges, recurrent heads]
//   | [branch norms and gates + output projections] | [branch average, norms + gate|up] | [GLU + down]
// and per token the head with the arg-max. A cooperative grid stays resident over all tokens of a
// launch; every phase deals its rows (or its heads) to the CTAs, and while a CTA waits at a barrier
// the weights of a coming phase are on their way into L2. Vectors between phases are fp32; every CTA
// stages (and norms) its own copy. All waits are bounded.
#include <cfloat>

#include "decode_core.h"
#include "hybrid_kernels.h"
#include "hybrid_token.h"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int kThreads = 256, kWarps = 8;

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
};

// dot(W[row, part of K], xs) over a warp that owns the chunks part, part + WPR, ...: all lanes get the sum.
template <typename T>
__device__ __forceinline__ float row_dot(const T* __restrict__ row, const float* xs, int K, int part, int wpr) {
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
  return warp_sum(acc);
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
  float acc = 0.0f;
  for (int i = 0; i < n; i += Chunk<T>::kN) {
    Chunk<T> c;
    c.load(row + i);
    acc = c.dot(x + i, acc);
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

template <typename T>
__device__ void prefetch_phase(const TokenPhase& ph) {
  for (int s = 0; s < ph.n_gemv; ++s) {
    const TokenGemv& g = ph.gemv[s];
    const char* base = static_cast<const char*>(g.W);
    const int64_t lines = static_cast<int64_t>(g.rows) * g.K * sizeof(T) / 128;
    for (int64_t i = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x; i < lines; i += static_cast<int64_t>(gridDim.x) * kThreads)
      prefetch_l2(base + i * 128);
  }
}

template <typename T>
__global__ void __launch_bounds__(kThreads, 2) hybrid_token_kernel(const __grid_constant__ TokenArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ TokenPhase ph_s[2];
  __shared__ float red[2 * kWarps];
  __shared__ float part_red[kWarps];
  __shared__ unsigned long long best_s[kWarps];
  __shared__ int s_flag;
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
      if (ph.is_mix) {
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
        unsigned long long best = 0ull;
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
        if (ph.is_head && a.out_tokens != nullptr) {
          if (lane == 0) best_s[wid] = best;
          __syncthreads();
          if (threadIdx.x == 0) {
#pragma unroll
            for (int w = 1; w < kWarps; ++w) best = best_s[w] > best ? best_s[w] : best;
            atomicMax(&words[t & 1], best);
          }
        }
      }
      if (ph.prefetch >= 0) prefetch_phase<T>(a.phases[ph.prefetch]);
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
int token_grid(size_t smem, int* grid) {
  int dev = 0, coop = 0, per_sm = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e == cudaSuccess) e = cudaDeviceGetAttribute(&coop, cudaDevAttrCooperativeLaunch, dev);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(hybrid_token_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e == cudaSuccess) e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, hybrid_token_kernel<T>, kThreads, smem);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "hybrid token kernel: %s", cudaGetErrorString(e));
  CTDK_REQUIRE(coop != 0 && per_sm >= 1, "hybrid token kernel: no cooperative launch with %zu bytes of shared memory", smem);
  *grid = sm_count() * (per_sm > 2 ? 2 : per_sm);
  return CTDK_OK;
}

template <typename T>
int launch_token_kernel(const TokenArgs& a, int grid, size_t smem, cudaStream_t s) {
  if (cudaMemsetAsync(a.sync, 0, a.sync_words * sizeof(unsigned int), s) != cudaSuccess)
    return fail(CTDK_ELAUNCH, "hybrid token kernel: clearing the barrier words failed");
  TokenArgs args = a;
  void* params[] = {&args};
  const cudaError_t e = cudaLaunchCooperativeKernel(reinterpret_cast<const void*>(hybrid_token_kernel<T>), dim3(grid), dim3(kThreads),
                                                    params, smem, s);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "hybrid token kernel: %s", cudaGetErrorString(e));
  return check_launch("hybrid token kernel");
}

template int token_grid<float>(size_t, int*);
template int token_grid<__nv_bfloat16>(size_t, int*);
template int launch_token_kernel<float>(const TokenArgs&, int, size_t, cudaStream_t);
template int launch_token_kernel<__nv_bfloat16>(const TokenArgs&, int, size_t, cudaStream_t);

}  // namespace hybrid
}  // namespace ctdk
