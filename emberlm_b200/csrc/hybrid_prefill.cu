// Row-wise kernels of the layer-list family's prompt pass (hybrid_kernels.h): sandwich norms, the
// packing around chunked attention, short convolutions and gates of the delta rule.
#include <cfloat>

#include "hybrid_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

int row_grid(int64_t rows, int per_cta = 1) {
  const int64_t need = (rows + per_cta - 1) / per_cta, cap = static_cast<int64_t>(sm_count()) * 16;
  return static_cast<int>(need < cap ? need : cap);
}

// Block-wide sums of N values (blockDim 256); two slots so that one barrier per reduction suffices.
template <int N>
__device__ __forceinline__ void block_sum(float (&v)[N], float* smem /* [2][N][8] */, int& slot) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  float* s = smem + slot * N * 8;
  slot ^= 1;
#pragma unroll
  for (int k = 0; k < N; ++k) {
    v[k] = warp_sum(v[k]);
    if (lane == 0) s[k * 8 + wid] = v[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < N; ++k) {
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) t += s[k * 8 + i];
    v[k] = t;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) norm_rows_kernel(const NormArgs<T> a, int64_t rows) {
  extern __shared__ float row_s[];   // [width] y, [width] x
  __shared__ float red[2 * 2 * 8];
  pdl_launch();
  pdl_wait();
  float* ys = row_s;
  float* xs = row_s + a.width;
  int slot = 0;
  const int W = a.width;
  const float inv = 1.0f / static_cast<float>(W);
  // every thread only ever touches its own columns (tid, tid + 256, ...) of ys / xs
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    const int64_t src = a.gather != nullptr ? a.gather[r] : r;
    float ss[2] = {0.0f, 0.0f};
    if (a.ids != nullptr) {
      const T* e = a.embed + a.ids[src] * a.ld_embed;
      for (int i = threadIdx.x; i < W; i += 256) {
        const float v = to_f(e[i]);
        ys[i] = v;
        ss[0] += v * v;
      }
      block_sum<2>(ss, red, slot);
      const float sc = rsqrtf(ss[0] * inv + a.eps);
      for (int i = threadIdx.x; i < W; i += 256) xs[i] = ys[i] * sc * a.w_embed[i];
    } else {
      const float* y = a.y + src * W;
      if (a.y2 != nullptr) {
        const float* y2 = a.y2 + src * W;
        for (int i = threadIdx.x; i < W; i += 256) {
          const float u = y[i], v = y2[i];
          ys[i] = u;
          xs[i] = v;
          ss[0] += u * u;
          ss[1] += v * v;
        }
        block_sum<2>(ss, red, slot);
        const float s1 = rsqrtf(ss[0] * inv + a.eps), s2 = rsqrtf(ss[1] * inv + a.eps);
        ss[0] = ss[1] = 0.0f;
        for (int i = threadIdx.x; i < W; i += 256) {
          const float v = 0.5f * (ys[i] * s1 * a.w_y[i] + xs[i] * s2 * a.w_y2[i]);
          ys[i] = v;
          ss[0] += v * v;
        }
      } else {
        for (int i = threadIdx.x; i < W; i += 256) {
          const float v = y[i];
          ys[i] = v;
          ss[0] += v * v;
        }
      }
      block_sum<2>(ss, red, slot);
      const float sc = rsqrtf(ss[0] * inv + a.eps);
      const float* x = a.x + src * W;
      for (int i = threadIdx.x; i < W; i += 256) xs[i] = x[i] + ys[i] * sc * a.w_post[i];
    }
    ss[0] = 0.0f;
    for (int i = threadIdx.x; i < W; i += 256) {
      const float v = xs[i];
      if (a.x_out != nullptr) a.x_out[r * W + i] = v;
      ss[0] += v * v;
    }
    block_sum<2>(ss, red, slot);
    const float sc = rsqrtf(ss[0] * inv + a.eps);
    for (int i = threadIdx.x; i < W; i += 256) a.h[r * a.ld_h + i] = from_f<T>(xs[i] * sc * a.w_pre[i]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
    clamped_glu_kernel(const float* __restrict__ gu, T* __restrict__ act, int64_t rows, int ffp, float limit) {
  pdl_launch();
  pdl_wait();
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    const float* g_row = gu + r * 2 * ffp;
#pragma unroll 4
    for (int c = threadIdx.x * 4; c < ffp; c += 1024) {
      const float4 g = load4(g_row + c), u = load4(g_row + ffp + c);
      store4(act + r * ffp + c, make_float4(clamped_glu_f(g.x, u.x, limit), clamped_glu_f(g.y, u.y, limit),
                                            clamped_glu_f(g.z, u.z, limit), clamped_glu_f(g.w, u.w, limit)));
    }
  }
}

__global__ void __launch_bounds__(256) rope_table_f64_kernel(float2* table, int64_t n, const double* freqs, int pairs) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= n * pairs) return;
  double sn, cs;
  sincos(static_cast<double>(i / pairs) * freqs[i % pairs], &sn, &cs);
  table[i] = make_float2(static_cast<float>(cs), static_cast<float>(sn));
}

// One thread per (row, head, column pair).
template <typename T>
__global__ void __launch_bounds__(256) attn_pack_kernel(const AttnArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int P = a.Dp / 2, heads = a.H + a.G, RS = (a.H + 2 * a.G) * a.Dp;
  const int64_t n = rows * heads * P, stride = static_cast<int64_t>(gridDim.x) * 256;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += stride) {
    const int p = static_cast<int>(i % P);
    const int hh = static_cast<int>((i / P) % heads);
    const int64_t r = i / (static_cast<int64_t>(P) * heads);
    const bool is_q = hh < a.H;
    const int head = is_q ? hh : hh - a.H, d = 2 * p;
    float u = 0.0f, v = 0.0f;
    if (r >= first) {
      const float* src = a.proj + (r - first) * a.ldp + (is_q ? a.col_q : a.col_k) + head * a.dim;
      const float* bias = (is_q ? a.b_q : a.b_k) + head * a.dim;
      if (d < a.dim) u = src[d] + bias[d];
      if (d + 1 < a.dim) v = src[d + 1] + bias[d + 1];
    } else if (!is_q) {
      const T* src = a.cache + (static_cast<int64_t>(head) * a.chunk + r) * a.dim;
      if (d < a.dim) u = to_f(src[d]);
      if (d + 1 < a.dim) v = to_f(src[d + 1]);
    }
    float* dst = a.packed + r * RS + d;
    if (!is_q) *reinterpret_cast<float2*>(dst + (a.H + a.G + head) * a.Dp) = make_float2(u, v);
    float2 o = make_float2(u, v);
    if (p < a.rot_pairs) {
      const float2 cs = a.table[(r % a.chunk) * a.rot_pairs + p];
      o = make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
    }
    *reinterpret_cast<float2*>(dst + hh * a.Dp) = o;
  }
}

// The same for head sizes that are multiples of four: four columns per thread, a row per CTA turn.
template <typename T>
__global__ void __launch_bounds__(256) attn_pack4_kernel(const AttnArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int P = a.Dp / 4, heads = a.H + a.G, RS = (a.H + 2 * a.G) * a.Dp, n = heads * P;
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    const bool fresh = r >= first;
    const float* row = a.proj + (r - first) * a.ldp;
    const float2* table = a.table + (r % a.chunk) * a.rot_pairs;
    float* out = a.packed + r * RS;
#pragma unroll 2
    for (int i = threadIdx.x; i < n; i += 256) {
      const int hh = i / P, d = (i % P) * 4;
      const bool is_q = hh < a.H;
      const int head = is_q ? hh : hh - a.H;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d < a.dim) {
        if (fresh) {
          x = load4(row + (is_q ? a.col_q : a.col_k) + head * a.dim + d);
          const float4 b = load4((is_q ? a.b_q : a.b_k) + head * a.dim + d);
          x.x += b.x;
          x.y += b.y;
          x.z += b.z;
          x.w += b.w;
        } else if (!is_q) {
          x = load4(a.cache + (static_cast<int64_t>(head) * a.chunk + r) * a.dim + d);
        }
      }
      if (!is_q) store4(out + (a.H + a.G + head) * a.Dp + d, x);
      const int p = d >> 1;
      if (p < a.rot_pairs) {
        const float2 cs = table[p];
        x = make_float4(x.x * cs.x - x.y * cs.y, x.y * cs.x + x.x * cs.y, x.z, x.w);
      }
      if (p + 1 < a.rot_pairs) {
        const float2 cs = table[p + 1];
        x = make_float4(x.x, x.y, x.z * cs.x - x.w * cs.y, x.w * cs.x + x.z * cs.y);
      }
      store4(out + hh * a.Dp + d, x);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) attn_store_kernel(const AttnArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int64_t base = (rows - 1) / a.chunk * a.chunk, from = base > first ? base : first;
  const int cols = a.G * a.dim;
  const int64_t n = (rows - from) * cols, stride = static_cast<int64_t>(gridDim.x) * 256;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += stride) {
    const int c = static_cast<int>(i % cols);
    const int64_t r = from + i / cols;
    const int g = c / a.dim, d = c % a.dim;
    a.cache[(static_cast<int64_t>(g) * a.chunk + (r - base)) * a.dim + d] =
        from_f<T>(a.proj[(r - first) * a.ldp + a.col_k + c] + a.b_k[c]);
  }
}

// One warp per (query row, head); lanes walk the keys for the scores and the columns for the output.
__global__ void __launch_bounds__(256)
    attn_chunked_fp32_kernel(const float* __restrict__ packed, float* __restrict__ out, int64_t first, int64_t rows, int64_t chunk,
                             int H, int G, int dim, int Dp, float scale) {
  extern __shared__ float qs_all[];   // [8][dim]
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  float* qs = qs_all + wid * dim;
  const int RS = (H + 2 * G) * Dp;
  const int64_t n = (rows - first) * H;
  for (int64_t it = static_cast<int64_t>(blockIdx.x) * 8 + wid; it < n; it += static_cast<int64_t>(gridDim.x) * 8) {
    const int h = static_cast<int>(it % H), g = h / (H / G);
    const int64_t r = first + it / H, j0 = r / chunk * chunk;
    __syncwarp();
    for (int d = lane; d < dim; d += 32) qs[d] = packed[r * RS + h * Dp + d];
    __syncwarp();
    const float* kb = packed + (H + g) * Dp;
    const float* vb = packed + (H + G + g) * Dp;
    float m = -FLT_MAX, l = 0.0f;
    float acc[32];
#pragma unroll
    for (int c = 0; c < 32; ++c) acc[c] = 0.0f;
    for (int64_t jb = j0; jb <= r; jb += 32) {
      const int64_t j = jb + lane;
      float sc = -FLT_MAX;
      if (j <= r) {
        const float* kr = kb + j * RS;
        float t = 0.0f;
        for (int d = 0; d < dim; ++d) t = fmaf(qs[d], kr[d], t);
        sc = t * scale;
      }
      const float mn = fmaxf(m, warp_max(sc));
      const float p = j <= r ? expf(sc - mn) : 0.0f;
      const float c0 = expf(m - mn);
      l = l * c0 + warp_sum(p);
      m = mn;
      const int nk = static_cast<int>(r - jb + 1 < 32 ? r - jb + 1 : 32);
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        const int d = lane + 32 * c;
        if (32 * c < dim) {
          float t = acc[c] * c0;
          for (int u = 0; u < nk; ++u) {
            const float pu = __shfl_sync(0xffffffffu, p, u);
            if (d < dim) t = fmaf(pu, vb[(jb + u) * RS + d], t);
          }
          acc[c] = t;
        }
      }
    }
    const float inv = 1.0f / l;
#pragma unroll
    for (int c = 0; c < 32; ++c) {
      const int d = lane + 32 * c;
      if (d < dim) out[r * H * Dp + h * Dp + d] = acc[c] * inv;
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) attn_gate_kernel(const AttnArgs<T> a, T* dst, int64_t ld, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int cols = a.H * a.dim;
  const int64_t n = (rows - first) * cols, stride = static_cast<int64_t>(gridDim.x) * 256;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += stride) {
    const int c = static_cast<int>(i % cols);
    const int64_t t = i / cols;
    const int h = c / a.dim, d = c % a.dim;
    dst[t * ld + c] = from_f<T>(a.out[(first + t) * a.H * a.Dp + h * a.Dp + d] * sigmoid_f(a.proj[t * a.ldp + a.col_g + h]));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) attn_gate4_kernel(const AttnArgs<T> a, T* dst, int64_t ld, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int P = a.dim / 4, n = a.H * P;
  for (int64_t t = blockIdx.x; t < rows - first; t += gridDim.x) {
    const float* o = a.out + (first + t) * a.H * a.Dp;
    const float* g = a.proj + t * a.ldp + a.col_g;
#pragma unroll 2
    for (int i = threadIdx.x; i < n; i += 256) {
      const int h = i / P, d = (i % P) * 4;
      const float4 v = load4(o + h * a.Dp + d);
      const float s = sigmoid_f(g[h]);
      store4(dst + t * ld + h * a.dim + d, make_float4(v.x * s, v.y * s, v.z * s, v.w * s));
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, const float* __restrict__ w,
                                                         const float* __restrict__ gate, int64_t ldg, T* __restrict__ dst, int64_t ld,
                                                         int64_t rows, int n, float eps) {
  __shared__ float red[2 * 8];
  pdl_launch();
  pdl_wait();
  int slot = 0;
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    float ss[1] = {0.0f};
    for (int i = threadIdx.x; i < n; i += 256) {
      const float v = o[r * n + i];
      ss[0] += v * v;
    }
    block_sum<1>(ss, red, slot);
    const float sc = rsqrtf(ss[0] / static_cast<float>(n) + eps);
    for (int i = threadIdx.x; i < n; i += 256)
      dst[r * ld + i] = from_f<T>(o[r * n + i] * sc * w[i] * sigmoid_f(gate[r * ldg + i]));
  }
}

// One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
    gated_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, const float* __restrict__ gate, int64_t ldg,
                           T* __restrict__ dst, int64_t ld, int64_t rows, int H, int vdim, float eps) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t nw = static_cast<int64_t>(gridDim.x) * 8;
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < rows * H; i += nw) {
    const int64_t r = i / H;
    const int h = static_cast<int>(i % H);
    const float* x = o + i * vdim;
    float ss = 0.0f;
    for (int d = lane; d < vdim; d += 32) ss += x[d] * x[d];
    const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(vdim) + eps);
    for (int d = lane; d < vdim; d += 32)
      dst[r * ld + h * vdim + d] = from_f<T>(x[d] * sc * w[d] * sigmoid_f(gate[r * ldg + h * vdim + d]));
  }
}

// Convolved and activated channel c (of the concatenated q | k | v channels) at portion row t.
__device__ __forceinline__ float conv_silu(const DeltaPrepArgs& a, int64_t t, int col, const float* taps, int c, int ring_c, int ring_ld) {
  float y = 0.0f;
  for (int j = 0; j < a.taps; ++j) {
    const int64_t src = t - (a.taps - 1) + j;
    float x;
    if (src >= 0) {
      x = a.proj[src * a.ldp + col + c];
    } else {
      const int64_t p = a.pos + src;
      if (p < 0) continue;
      x = a.ring[(p % a.taps) * ring_ld + ring_c];
    }
    y = fmaf(taps[static_cast<int64_t>(c) * a.taps + j], x, y);
  }
  return silu_f(y);
}

// One warp per (row, unit); units: G q heads, G k heads, H v heads, H decay heads.
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaPrepArgs a) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int units = 2 * a.G + 2 * a.H, qk = a.G * a.dim, ring_ld = 2 * qk + a.H * a.vdim;
  const int64_t n = a.rows * units, nw = static_cast<int64_t>(gridDim.x) * 8;
  const float qscale = rsqrtf(static_cast<float>(a.dim));
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < n; i += nw) {
    const int64_t t = i / units;
    const int u = static_cast<int>(i % units);
    if (u < 2 * a.G) {
      const bool is_q = u < a.G;
      const int head = is_q ? u : u - a.G;
      float y[8];   // dim <= 256
      float ss = 0.0f;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int d = lane + 32 * e;
        y[e] = 0.0f;
        if (d < a.dim) {
          const int c = head * a.dim + d;
          y[e] = is_q ? conv_silu(a, t, a.col_q, a.conv_q, c, c, ring_ld) : conv_silu(a, t, a.col_k, a.conv_k, c, qk + c, ring_ld);
          ss += y[e] * y[e];
        }
      }
      const float sc = rsqrtf(warp_sum(ss) + 1e-6f) * (is_q ? qscale : 1.0f);
      float* dst = (is_q ? a.q : a.k) + t * qk + head * a.dim;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int d = lane + 32 * e;
        if (d < a.dim) dst[d] = y[e] * sc;
      }
    } else if (u < 2 * a.G + a.H) {
      const int head = u - 2 * a.G;
      for (int d = lane; d < a.vdim; d += 32) {
        const int c = head * a.vdim + d;
        a.v[t * a.H * a.vdim + c] = conv_silu(a, t, a.col_v, a.conv_v, c, 2 * qk + c, ring_ld);
      }
    } else {
      const int head = u - 2 * a.G - a.H;
      const float amp = -expf(a.a_log[head]);
      for (int d = lane; d < a.dim; d += 32) {
        const int c = head * a.dim + d;
        a.logg[t * a.H * a.dim + c] = amp * softplus_f(a.z[t * a.ldz + c] + a.dt_bias[c]);
      }
      if (lane == 0) a.beta[t * a.H + head] = sigmoid_f(a.proj[t * a.ldp + a.col_b + head]);
    }
  }
}

// The same for four taps with a sliding window: one warp per (unit, run of kRun rows), so that a
// projection row is read once. E = ceil(max(dim, vdim) / 32) channels per lane.
constexpr int kRun = 8, kAhead = 4;
template <int E>
__global__ void __launch_bounds__(256, 3) delta_prep4_kernel(const DeltaPrepArgs a) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int units = 2 * a.G + 2 * a.H, qk = a.G * a.dim, ring_ld = 2 * qk + a.H * a.vdim;
  const int64_t runs = (a.rows + kRun - 1) / kRun, n = runs * units, nw = static_cast<int64_t>(gridDim.x) * 8;
  const float qscale = rsqrtf(static_cast<float>(a.dim));
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < n; i += nw) {
    const int u = static_cast<int>(i % units);
    const int64_t t0 = i / units * kRun, t1 = t0 + kRun < a.rows ? t0 + kRun : a.rows;
    if (u >= 2 * a.G + a.H) {   // decays and beta
      const int head = u - 2 * a.G - a.H;
      const float amp = -expf(a.a_log[head]);
      for (int d = lane; d < a.dim; d += 32) {
        const int c = head * a.dim + d;
        const float bias = a.dt_bias[c];
        float z[kRun];
#pragma unroll
        for (int r = 0; r < kRun; ++r) z[r] = t0 + r < t1 ? a.z[(t0 + r) * a.ldz + c] : 0.0f;
#pragma unroll
        for (int r = 0; r < kRun; ++r)
          if (t0 + r < t1) a.logg[(t0 + r) * a.H * a.dim + c] = amp * softplus_f(z[r] + bias);
      }
      if (t0 + lane < t1) a.beta[(t0 + lane) * a.H + head] = sigmoid_f(a.proj[(t0 + lane) * a.ldp + a.col_b + head]);
      continue;
    }
    const int kind = u < a.G ? 0 : (u < 2 * a.G ? 1 : 2);
    const int head = kind == 0 ? u : (kind == 1 ? u - a.G : u - 2 * a.G);
    const int width = kind == 2 ? a.vdim : a.dim;
    const int col = (kind == 0 ? a.col_q : (kind == 1 ? a.col_k : a.col_v)) + head * width;
    const int ring_c = (kind == 0 ? 0 : (kind == 1 ? qk : 2 * qk)) + head * width;
    const float* taps = (kind == 0 ? a.conv_q : (kind == 1 ? a.conv_k : a.conv_v)) + static_cast<int64_t>(head) * width * 4;
    float4 w[E];
    float x0[E], x1[E], x2[E];   // inputs three, two and one rows back
    auto before = [&](int64_t t, int d) {
      if (t >= 0) return a.proj[t * a.ldp + col + d];
      const int64_t p = a.pos + t;
      return p < 0 ? 0.0f : a.ring[(p & 3) * ring_ld + ring_c + d];
    };
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int d = lane + 32 * e;
      w[e] = make_float4(0.f, 0.f, 0.f, 0.f);
      x0[e] = x1[e] = x2[e] = 0.0f;
      if (d < width) {
        w[e] = *reinterpret_cast<const float4*>(taps + static_cast<int64_t>(d) * 4);
        x0[e] = before(t0 - 3, d);
        x1[e] = before(t0 - 2, d);
        x2[e] = before(t0 - 1, d);
      }
    }
#pragma unroll 1
    for (int64_t tb = t0; tb < t1; tb += kAhead) {
      float rows_x[kAhead][E];   // requested together
#pragma unroll
      for (int r = 0; r < kAhead; ++r)
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const int d = lane + 32 * e;
          rows_x[r][e] = (d < width && tb + r < t1) ? a.proj[(tb + r) * a.ldp + col + d] : 0.0f;
        }
#pragma unroll
      for (int r = 0; r < kAhead; ++r) {
        const int64_t t = tb + r;
        if (t >= t1) break;
        float y[E], ss = 0.0f;
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const float x = rows_x[r][e];
          y[e] = silu_f(fmaf(w[e].w, x, fmaf(w[e].z, x2[e], fmaf(w[e].y, x1[e], w[e].x * x0[e]))));
          ss += y[e] * y[e];
          x0[e] = x1[e];
          x1[e] = x2[e];
          x2[e] = x;
        }
        float sc = 1.0f;
        if (kind < 2) sc = rsqrtf(warp_sum(ss) + 1e-6f) * (kind == 0 ? qscale : 1.0f);
        float* dst = kind == 2 ? a.v + t * a.H * a.vdim + head * width : (kind == 0 ? a.q : a.k) + t * qk + head * width;
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const int d = lane + 32 * e;
          if (d < width) dst[d] = y[e] * sc;
        }
      }
    }
  }
}

__global__ void __launch_bounds__(256) delta_ring_store_kernel(const DeltaPrepArgs a) {
  pdl_launch();
  pdl_wait();
  const int qk = a.G * a.dim, ring_ld = 2 * qk + a.H * a.vdim;
  const int64_t keep = a.rows < a.taps ? a.rows : a.taps;
  const int64_t n = keep * ring_ld, stride = static_cast<int64_t>(gridDim.x) * 256;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += stride) {
    const int64_t t = a.rows - keep + i / ring_ld;
    const int c = static_cast<int>(i % ring_ld);
    const int col = c < qk ? a.col_q + c : (c < 2 * qk ? a.col_k + c - qk : a.col_v + c - 2 * qk);
    a.ring[((a.pos + t) % a.taps) * ring_ld + c] = a.proj[t * a.ldp + col];
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
    cast_columns_kernel(const float* __restrict__ src, int64_t lds, T* __restrict__ dst, int64_t ldd, int64_t rows, int cols) {
  pdl_launch();
  pdl_wait();
  const int64_t n = rows * cols, stride = static_cast<int64_t>(gridDim.x) * 256;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += stride) {
    const int64_t r = i / cols;
    const int c = static_cast<int>(i % cols);
    dst[r * ldd + c] = from_f<T>(src[r * lds + c]);
  }
}

#define LAUNCH(what, kernel, grid, smem, ...)                                                                    \
  do {                                                                                                           \
    const cudaError_t e_ = launch_pdl(kernel, dim3(grid), dim3(256), smem, s, __VA_ARGS__);                      \
    if (e_ != cudaSuccess) return fail(CTDK_ELAUNCH, what ": %s", cudaGetErrorString(e_));                       \
    return check_launch(what);                                                                                   \
  } while (0)

}  // namespace

template <typename T>
int norm_rows(const NormArgs<T>& a, int64_t rows, cudaStream_t s) {
  if (rows == 0) return CTDK_OK;
  const size_t smem = static_cast<size_t>(a.width) * 8;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(norm_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "hybrid norm: %s", cudaGetErrorString(e));
  }
  LAUNCH("hybrid norm", norm_rows_kernel<T>, row_grid(rows), smem, a, rows);
}
template <typename T>
int clamped_glu_rows(const float* gu, T* act, int64_t rows, int ffp, float limit, cudaStream_t s) {
  LAUNCH("hybrid glu", clamped_glu_kernel<T>, row_grid(rows), 0, gu, act, rows, ffp, limit);
}
int rope_table_f64(float2* table, int64_t n, const double* freqs_dev, int pairs, cudaStream_t s) {
  rope_table_f64_kernel<<<ceil_div(n * pairs, 256), 256, 0, s>>>(table, n, freqs_dev, pairs);
  return check_launch("hybrid rope table");
}
template <typename T>
int attn_pack(const AttnArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s) {
  if (a.dim % 4 == 0) LAUNCH("hybrid attention pack", attn_pack4_kernel<T>, row_grid(rows), 0, a, first, rows);
  LAUNCH("hybrid attention pack", attn_pack_kernel<T>, row_grid(rows * (a.H + a.G) * (a.Dp / 2), 256), 0, a, first, rows);
}
template <typename T>
int attn_store(const AttnArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s) {
  const int64_t most = rows - first < a.chunk ? rows - first : a.chunk;
  LAUNCH("hybrid key store", attn_store_kernel<T>, row_grid(most * a.G * a.dim, 256), 0, a, first, rows);
}
int attn_chunked_fp32(const float* packed, float* out, int64_t first, int64_t rows, int64_t chunk, int H, int G, int dim, int Dp,
                      float scale, cudaStream_t s) {
  CTDK_REQUIRE(dim <= 1024, "hybrid attention: head size above 1024");
  attn_chunked_fp32_kernel<<<row_grid((rows - first) * H, 8), 256, static_cast<size_t>(8) * dim * 4, s>>>(packed, out, first, rows, chunk,
                                                                                                     H, G, dim, Dp, scale);
  return check_launch("hybrid attention (fp32)");
}
template <typename T>
int attn_gate(const AttnArgs<T>& a, T* dst, int64_t ld, int64_t first, int64_t rows, cudaStream_t s) {
  if (a.dim % 4 == 0) LAUNCH("hybrid attention gate", attn_gate4_kernel<T>, row_grid(rows - first), 0, a, dst, ld, first, rows);
  LAUNCH("hybrid attention gate", attn_gate_kernel<T>, row_grid((rows - first) * a.H * a.dim, 256), 0, a, dst, ld, first, rows);
}
template <typename T>
int gated_norm_rows(const float* o, const float* w, const float* gate, int64_t ldg, T* dst, int64_t ld, int64_t rows, int n, float eps,
                    cudaStream_t s) {
  LAUNCH("hybrid gated norm", gated_norm_kernel<T>, row_grid(rows), 0, o, w, gate, ldg, dst, ld, rows, n, eps);
}
template <typename T>
int gated_head_norm_rows(const float* o, const float* w, const float* gate, int64_t ldg, T* dst, int64_t ld, int64_t rows, int H,
                         int vdim, float eps, cudaStream_t s) {
  LAUNCH("hybrid head norm", gated_head_norm_kernel<T>, row_grid(rows * H, 8), 0, o, w, gate, ldg, dst, ld, rows, H, vdim, eps);
}
int delta_prep(const DeltaPrepArgs& a, cudaStream_t s) {
  const int wide = a.dim > a.vdim ? a.dim : a.vdim;
  if (a.taps == 4 && wide <= 128) {
    const int grid = row_grid((a.rows + kRun - 1) / kRun * (2 * a.G + 2 * a.H), 8);
    if (wide <= 32) LAUNCH("delta prep", delta_prep4_kernel<1>, grid, 0, a);
    if (wide <= 64) LAUNCH("delta prep", delta_prep4_kernel<2>, grid, 0, a);
    LAUNCH("delta prep", delta_prep4_kernel<4>, grid, 0, a);
  }
  LAUNCH("delta prep", delta_prep_kernel, row_grid(a.rows * (2 * a.G + 2 * a.H), 8), 0, a);
}
int delta_ring_store(const DeltaPrepArgs& a, cudaStream_t s) {
  LAUNCH("delta ring", delta_ring_store_kernel, row_grid(static_cast<int64_t>(a.taps) * (2 * a.G * a.dim + a.H * a.vdim), 256), 0, a);
}
template <typename T>
int cast_columns(const float* src, int64_t lds, T* dst, int64_t ldd, int64_t rows, int cols, cudaStream_t s) {
  LAUNCH("hybrid cast", cast_columns_kernel<T>, row_grid(rows * cols, 256), 0, src, lds, dst, ldd, rows, cols);
}

#define INSTANTIATE(T)                                                                                                              \
  template int norm_rows<T>(const NormArgs<T>&, int64_t, cudaStream_t);                                                             \
  template int clamped_glu_rows<T>(const float*, T*, int64_t, int, float, cudaStream_t);                                            \
  template int attn_pack<T>(const AttnArgs<T>&, int64_t, int64_t, cudaStream_t);                                                    \
  template int attn_store<T>(const AttnArgs<T>&, int64_t, int64_t, cudaStream_t);                                                   \
  template int attn_gate<T>(const AttnArgs<T>&, T*, int64_t, int64_t, int64_t, cudaStream_t);                                       \
  template int gated_norm_rows<T>(const float*, const float*, const float*, int64_t, T*, int64_t, int64_t, int, float, cudaStream_t); \
  template int gated_head_norm_rows<T>(const float*, const float*, const float*, int64_t, T*, int64_t, int64_t, int, int, float,    \
                                       cudaStream_t);                                                                               \
  template int cast_columns<T>(const float*, int64_t, T*, int64_t, int64_t, int, cudaStream_t);
INSTANTIATE(float)
INSTANTIATE(__nv_bfloat16)

}  // namespace hybrid
}  // namespace ctdk
