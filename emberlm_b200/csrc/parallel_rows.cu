// Row-wise kernels of the parallel arrangement's prompt pass (parallel_kernels.h).
#include "hybrid_kernels.h"
#include "parallel_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

int row_grid(int64_t rows, int per_cta = 1) {
  const int64_t need = (rows + per_cta - 1) / per_cta, cap = static_cast<int64_t>(sm_count()) * 16;
  return static_cast<int>(need < cap ? need : cap);
}

template <int V>
struct Vec {
  float v[V];
};
template <int V, typename U>
__device__ __forceinline__ Vec<V> vload(const U* p) {
  Vec<V> r;
  if constexpr (V == 4) {
    const float4 f = load4(p);
    r.v[0] = f.x;
    r.v[1] = f.y;
    r.v[2] = f.z;
    r.v[3] = f.w;
  } else {
    r.v[0] = to_f(*p);
  }
  return r;
}
template <int V, typename U>
__device__ __forceinline__ void vstore(U* p, const Vec<V>& r) {
  if constexpr (V == 4) store4(p, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
  else *p = from_f<U>(r.v[0]);
}

// A CTA walks `run` consecutive rows and keeps the previous row's h and m in shared memory; the one or two
// rows in front of its run are formed again (h needs one row back, a mix of shifted rows two). Columns are
// dealt so that a warp's columns lie in one group: wpg warps per group.
template <typename T, int V>
__global__ void __launch_bounds__(256, 4) shift_norm_kernel(const ShiftNormArgs<T> a, int64_t rows, int run, int wpg) {
  extern __shared__ __align__(16) float sm[];
  const int W = a.width, gs = W / a.groups, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int Wp = (W + 3) & ~3;
  float *xs = sm, *hs = xs + Wp, *ms = hs + Wp;
  float* part = a.shift == nullptr ? hs : (a.n_mix > 0 ? ms + Wp : ms);   // [2][groups][wpg]
  pdl_launch();
  pdl_wait();
  const int64_t t0 = static_cast<int64_t>(blockIdx.x) * run, t1 = t0 + run < rows ? t0 + run : rows;
  const int halo = a.n_mix > 0 ? 2 : (a.shift != nullptr ? 1 : 0);
  const int g0 = wid / wpg, gstep = 8 / wpg, wj = wid % wpg;
  const bool active = g0 < gstep;
  const float inv = 1.0f / static_cast<float>(gs);
  int slot = 0;
  for (int64_t r = t0 - halo > 0 ? t0 - halo : 0; r < t1; ++r) {
    const bool own = r >= t0, have = r > 0 && r > t0 - halo;   // have: the previous row is in shared memory
    const int64_t src = a.gather != nullptr ? a.gather[r] : r;
    const T* e = a.ids != nullptr ? a.embed + a.ids[src] * a.ld_embed : nullptr;
    float* ps = part + slot * a.groups * wpg;
    slot ^= 1;
    for (int g = g0; active && g < a.groups; g += gstep) {
      float ss = 0.0f;
      for (int c = g * gs + (wj * 32 + lane) * V; c < (g + 1) * gs; c += 32 * V * wpg) {
        Vec<V> x;
        if (e != nullptr) {
          x = vload<V>(e + c);
#pragma unroll
          for (int k = 0; k < V; ++k) x.v[k] *= a.scale;
        } else {
          x = vload<V>(a.x + src * W + c);
          const Vec<V> y = vload<V>(a.y1 + src * W + c), z = vload<V>(a.z1 + src * a.ldz + c), b = vload<V>(a.b1 + c);
          Vec<V> y2, z2, b2;
          if (a.y2 != nullptr) {
            y2 = vload<V>(a.y2 + src * W + c);
            z2 = vload<V>(a.z2 + src * a.ldz + c);
            b2 = vload<V>(a.b2 + c);
          }
#pragma unroll
          for (int k = 0; k < V; ++k) {
            float u = y.v[k] * sigmoid_f(z.v[k] + b.v[k]);
            if (a.y2 != nullptr) u += y2.v[k] * sigmoid_f(z2.v[k] + b2.v[k]);
            x.v[k] += u;
          }
        }
#pragma unroll
        for (int k = 0; k < V; ++k) ss += x.v[k] * x.v[k];
        vstore<V>(xs + c, x);
        if (own && a.x_out != nullptr) vstore<V>(a.x_out + r * W + c, x);
      }
      ss = warp_sum(ss);
      if (lane == 0) ps[g * wpg + wj] = ss;
    }
    if (wpg > 1) __syncthreads();
    else __syncwarp();
    for (int g = g0; active && g < a.groups; g += gstep) {
      float ss = 0.0f;
      for (int k = 0; k < wpg; ++k) ss += ps[g * wpg + k];
      const float sc = rsqrtf(ss * inv + a.eps);
      for (int c = g * gs + (wj * 32 + lane) * V; c < (g + 1) * gs; c += 32 * V * wpg) {
        Vec<V> h = vload<V>(xs + c);
        const Vec<V> w = vload<V>(a.w + c);
#pragma unroll
        for (int k = 0; k < V; ++k) h.v[k] *= sc * w.v[k];
        if (own) vstore<V>(a.h + r * a.ld_h + c, h);
        if (a.shift == nullptr) continue;
        Vec<V> p;
#pragma unroll
        for (int k = 0; k < V; ++k) p.v[k] = 0.0f;
        if (have) p = vload<V>(hs + c);
        else if (r == 0 && a.prev_h != nullptr) p = vload<V>(a.prev_h + c);
        const Vec<V> f = vload<V>(a.shift + c);
        vstore<V>(hs + c, h);
        Vec<V> m;
#pragma unroll
        for (int k = 0; k < V; ++k) m.v[k] = fmaf(p.v[k] - h.v[k], f.v[k], h.v[k]);
        if (own) vstore<V>(a.shifted + r * a.ld_h + c, m);
        if (r == rows - 1) vstore<V>(a.next_h + c, h);
        if (a.n_mix == 0) continue;
#pragma unroll
        for (int k = 0; k < V; ++k) p.v[k] = 0.0f;
        if (have) p = vload<V>(ms + c);
        else if (r == 0 && a.prev_m != nullptr) p = vload<V>(a.prev_m + c);
        vstore<V>(ms + c, m);
        if (r == rows - 1) vstore<V>(a.next_m + c, m);
        if (own)
#pragma unroll
          for (int i = 0; i < kMaxMixes; ++i) {
            if (i >= a.n_mix) break;
            const Vec<V> mu = vload<V>(a.mu[i] + c);
            Vec<V> o;
#pragma unroll
            for (int k = 0; k < V; ++k) o.v[k] = fmaf(p.v[k] - m.v[k], mu.v[k], m.v[k]);
            vstore<V>(a.mix + i * a.mix_stride + r * a.ld_h + c, o);
          }
      }
    }
  }
}

__global__ void __launch_bounds__(256) commit_shift_kernel(const float* next, float* state, int layers, int slot, int width) {
  pdl_launch();
  pdl_wait();
  const int64_t per = 2ll * width, n = layers * per;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += static_cast<int64_t>(gridDim.x) * 256)
    state[(i / per * 2 + slot) * per + i % per] = next[i];
}

template <typename T, bool GELU>
__global__ void __launch_bounds__(256) glu_kernel(const float* __restrict__ gu, int64_t ldg, T* __restrict__ act, int64_t lda, int64_t rows,
                                                  int ffp, const int32_t* rows_dev) {
  pdl_launch();
  pdl_wait();
  if (rows_dev != nullptr && *rows_dev < rows) rows = *rows_dev;
  const int per = ffp / 4;
  const int64_t n = rows * per;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += static_cast<int64_t>(gridDim.x) * 256) {
    const int64_t r = i / per;
    const int c = static_cast<int>(i % per) * 4;
    const float4 g = load4(gu + r * ldg + c), u = load4(gu + r * ldg + ffp + c);
    float4 o;
    if (GELU) o = make_float4(gelu_tanh_f(g.x) * u.x, gelu_tanh_f(g.y) * u.y, gelu_tanh_f(g.z) * u.z, gelu_tanh_f(g.w) * u.w);
    else o = make_float4(silu_f(g.x) * u.x, silu_f(g.y) * u.y, silu_f(g.z) * u.z, silu_f(g.w) * u.w);
    store4(act + r * lda + c, o);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) tanh_rows_kernel(const float* __restrict__ src, int64_t lds, T* __restrict__ dst, int64_t ldd,
                                                       int64_t rows, int n) {
  pdl_launch();
  pdl_wait();
  const int64_t total = rows * n;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < total; i += static_cast<int64_t>(gridDim.x) * 256) {
    const int64_t r = i / n;
    const int c = static_cast<int>(i % n);
    dst[r * ldd + c] = from_f<T>(tanhf(src[r * lds + c]));
  }
}
// One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
    silu_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, const float* __restrict__ gate, int64_t ldg,
                          T* __restrict__ dst, int64_t ld, int64_t rows, int H, int dim, float eps) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t nw = static_cast<int64_t>(gridDim.x) * 8;
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < rows * H; i += nw) {
    const int64_t r = i / H;
    const int h = static_cast<int>(i % H);
    const float* x = o + i * dim;
    float ss = 0.0f;
    for (int d = lane; d < dim; d += 32) ss += x[d] * x[d];
    const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(dim) + eps);
    for (int d = lane; d < dim; d += 32) {
      const int c = h * dim + d;
      dst[r * ld + c] = from_f<T>(x[d] * sc * w[c] * silu_f(gate[r * ldg + c]));
    }
  }
}

#define LAUNCH(what, kernel, grid, smem, ...)                                                                    \
  do {                                                                                                           \
    const cudaError_t e_ = launch_pdl(kernel, dim3(grid), dim3(256), smem, s, __VA_ARGS__);                      \
    if (e_ != cudaSuccess) return fail(CTDK_ELAUNCH, what ": %s", cudaGetErrorString(e_));                       \
    return check_launch(what);                                                                                   \
  } while (0)

template <typename T, int V>
int launch_shift_norm(const ShiftNormArgs<T>& a, int64_t rows, cudaStream_t s) {
  const int wpg = a.groups >= 8 ? 1 : 8 / a.groups;
  const int arrays = a.n_mix > 0 ? 3 : (a.shift != nullptr ? 2 : 1);
  const size_t smem = (static_cast<size_t>((a.width + 3) / 4 * 4) * arrays + 2 * static_cast<size_t>(a.groups) * wpg) * 4;
  const int64_t slots = static_cast<int64_t>(sm_count()) * 4;   // CTAs that run at once
  const int64_t run64 = rows >= slots / 2 ? (rows + slots - 1) / slots : 1;
  const int run = a.gather != nullptr ? 1 : (run64 > 16 ? 16 : static_cast<int>(run64));
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(shift_norm_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "shift norm: %s", cudaGetErrorString(e));
  }
  LAUNCH("shift norm", (shift_norm_kernel<T, V>), static_cast<unsigned>((rows + run - 1) / run), smem, a, rows, run, wpg);
}

}  // namespace

template <typename T>
int shift_norm_rows(const ShiftNormArgs<T>& a, int64_t rows, cudaStream_t s) {
  if (rows == 0) return CTDK_OK;
  CTDK_REQUIRE(a.groups > 0 && a.width % a.groups == 0, "shift norm: groups must divide the width");
  // four columns at once need every row pitch to keep them aligned
  return a.width % (4 * a.groups) == 0 && a.ldz % 4 == 0 ? launch_shift_norm<T, 4>(a, rows, s) : launch_shift_norm<T, 1>(a, rows, s);
}
int commit_shift_state(const float* next, float* state, int layers, int slot, int width, cudaStream_t s) {
  LAUNCH("shift state", commit_shift_kernel, row_grid(2ll * layers * width, 256), 0, next, state, layers, slot, width);
}
template <typename T>
int glu_rows(const float* gu, int64_t ldg, T* act, int64_t lda, int64_t rows, int ffp, Glu kind, const int32_t* rows_dev, cudaStream_t s) {
  const int grid = row_grid(rows * (ffp / 4), 256);
  if (kind == Glu::kGelu) LAUNCH("gelu glu", (glu_kernel<T, true>), grid, 0, gu, ldg, act, lda, rows, ffp, rows_dev);
  LAUNCH("silu glu", (glu_kernel<T, false>), grid, 0, gu, ldg, act, lda, rows, ffp, rows_dev);
}
template <typename T>
int tanh_rows(const float* src, int64_t lds, T* dst, int64_t ldd, int64_t rows, int n, cudaStream_t s) {
  LAUNCH("tanh rows", tanh_rows_kernel<T>, row_grid(rows * n, 256), 0, src, lds, dst, ldd, rows, n);
}
template <typename T>
int silu_head_norm_rows(const float* o, const float* w, const float* gate, int64_t ldg, T* dst, int64_t ld, int64_t rows, int H, int dim,
                        float eps, cudaStream_t s) {
  LAUNCH("silu head norm", silu_head_norm_kernel<T>, row_grid(rows * H, 8), 0, o, w, gate, ldg, dst, ld, rows, H, dim, eps);
}

#define INSTANTIATE(T)                                                                                                               \
  template int shift_norm_rows<T>(const ShiftNormArgs<T>&, int64_t, cudaStream_t);                                                   \
  template int glu_rows<T>(const float*, int64_t, T*, int64_t, int64_t, int, Glu, const int32_t*, cudaStream_t);                     \
  template int tanh_rows<T>(const float*, int64_t, T*, int64_t, int64_t, int, cudaStream_t);                                         \
  template int silu_head_norm_rows<T>(const float*, const float*, const float*, int64_t, T*, int64_t, int64_t, int, int, float,      \
                                      cudaStream_t);
INSTANTIATE(float)
INSTANTIATE(__nv_bfloat16)

}  // namespace hybrid
}  // namespace ctdk
