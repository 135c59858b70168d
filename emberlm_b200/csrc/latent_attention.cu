// Latent attention of a prompt's portion: what lies around the attention product (norms of the down
// projections, rotation, cache rows) and the attention itself in fp32 for any size. Keys and values of every
// head have been read out of the cached latents into one buffer before; the rotated key part, shared by the
// heads, is taken from the cache. The tensor-core kernel is latent_attention_tc.cu.
#include <cfloat>

#include "hybrid_kernels.h"
#include "parallel_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

int row_grid(int64_t rows, int per_cta = 1) {
  const int64_t need = (rows + per_cta - 1) / per_cta, cap = static_cast<int64_t>(sm_count()) * 16;
  return static_cast<int>(need < cap ? need : cap);
}

// One warp per (row, query or key side).
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t nw = static_cast<int64_t>(gridDim.x) * 8;
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < 2 * rows; i += nw) {
    const int64_t r = i >> 1;
    const bool is_q = (i & 1) == 0;
    const int n = is_q ? a.q_rank : a.kv_rank;
    const float* x = a.proj + r * a.ldp + (is_q ? a.col_q : a.col_k);
    const float* w = is_q ? a.q_norm : a.kv_norm;
    T* dst = is_q ? a.low_q + r * a.ld_low : a.cache + (first + r) * a.ld_cache;
    float ss = 0.0f;
    for (int c = lane; c < n; c += 32) ss += x[c] * x[c];
    const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(n) + a.eps);
    for (int c = lane; c < n; c += 32) dst[c] = from_f<T>(x[c] * sc * w[c]);
    if (is_q) continue;
    const int half = a.rot_dim / 2;
    for (int p = lane; p < half; p += 32) {
      const float u = x[n + p], v = x[n + half + p];
      const float2 cs = a.table[(first + r) * half + p];
      dst[a.rot_col + p] = from_f<T>(u * cs.x - v * cs.y);
      dst[a.rot_col + half + p] = from_f<T>(v * cs.x + u * cs.y);
    }
  }
}

// The same for widths that are multiples of four: a row's side stays in registers, B float4 per lane.
template <typename T, int B>
__global__ void __launch_bounds__(256) latent_prep4_kernel(const LatentArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t nw = static_cast<int64_t>(gridDim.x) * 8;
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < 2 * rows; i += nw) {
    const int64_t r = i >> 1;
    const bool is_q = (i & 1) == 0;
    const int n = is_q ? a.q_rank : a.kv_rank;
    const float* x = a.proj + r * a.ldp + (is_q ? a.col_q : a.col_k);
    const float* w = is_q ? a.q_norm : a.kv_norm;
    T* dst = is_q ? a.low_q + r * a.ld_low : a.cache + (first + r) * a.ld_cache;
    float4 v[B];
    float ss = 0.0f;
#pragma unroll
    for (int u = 0; u < B; ++u) {
      const int c = (u * 32 + lane) * 4;
      v[u] = c < n ? load4(x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int u = 0; u < B; ++u) ss += v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
    const float sc = rsqrtf(warp_sum(ss) / static_cast<float>(n) + a.eps);
#pragma unroll
    for (int u = 0; u < B; ++u) {
      const int c = (u * 32 + lane) * 4;
      if (c < n) {
        const float4 g = load4(w + c);
        store4(dst + c, make_float4(v[u].x * sc * g.x, v[u].y * sc * g.y, v[u].z * sc * g.z, v[u].w * sc * g.w));
      }
    }
    if (is_q) continue;
    const int half = a.rot_dim / 2;
    for (int p = lane; p < half; p += 32) {
      const float u = x[n + p], y = x[n + half + p];
      const float2 cs = a.table[(first + r) * half + p];
      dst[a.rot_col + p] = from_f<T>(u * cs.x - y * cs.y);
      dst[a.rot_col + half + p] = from_f<T>(y * cs.x + u * cs.y);
    }
  }
}

// Head sizes that are multiples of eight and a rotated part of sixteen: a CTA per row, units of eight columns
// (unrotated) or of two times eight (the two halves of the rotated part).
template <typename T>
__global__ void __launch_bounds__(256) latent_rotate8_kernel(const LatentArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int D = a.dim + a.rot_dim, half = a.rot_dim / 2, flat = a.dim / 8, per = flat + half / 8, n = a.H * per;
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    const float* row = a.q_up + r * a.ld_up;
    const float2* table = a.table + (first + r) * half;
    T* out = a.q + r * a.H * D;
#pragma unroll 2
    for (int i = threadIdx.x; i < n; i += 256) {
      const int h = i / per, u = i % per;
      const int c = u < flat ? 8 * u : a.dim + 8 * (u - flat);
      const float* x = row + h * D + c;
      T* dst = out + h * D + c;
      const float4 p = load4(x), q = load4(x + 4);
      if (u < flat) {
        store4(dst, p);
        store4(dst + 4, q);
        continue;
      }
      const float4 s = load4(x + half), t = load4(x + half + 4);
      const float4* cs = reinterpret_cast<const float4*>(table + 8 * (u - flat));   // two pairs (cos, sin)
      const float4 c0 = cs[0], c1 = cs[1], c2 = cs[2], c3 = cs[3];
      store4(dst, make_float4(p.x * c0.x - s.x * c0.y, p.y * c0.z - s.y * c0.w, p.z * c1.x - s.z * c1.y, p.w * c1.z - s.w * c1.w));
      store4(dst + 4, make_float4(q.x * c2.x - t.x * c2.y, q.y * c2.z - t.y * c2.w, q.z * c3.x - t.z * c3.y, q.w * c3.z - t.w * c3.w));
      store4(dst + half, make_float4(s.x * c0.x + p.x * c0.y, s.y * c0.z + p.y * c0.w, s.z * c1.x + p.z * c1.y, s.w * c1.z + p.w * c1.w));
      store4(dst + half + 4, make_float4(t.x * c2.x + q.x * c2.y, t.y * c2.z + q.y * c2.w, t.z * c3.x + q.z * c3.y, t.w * c3.z + q.w * c3.w));
    }
  }
}

// One thread per (row, head, column of the padded head).
template <typename T>
__global__ void __launch_bounds__(256) latent_rotate_kernel(const LatentArgs<T> a, int64_t first, int64_t rows) {
  pdl_launch();
  pdl_wait();
  const int dp = (a.dim + 7) / 8 * 8, pitch = latent_q_pitch(a.dim, a.rot_dim), half = a.rot_dim / 2;
  const int64_t n = rows * a.H * pitch, stride = static_cast<int64_t>(gridDim.x) * 256;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n; i += stride) {
    const int c = static_cast<int>(i % pitch);
    const int64_t rh = i / pitch, r = rh / a.H;
    const float* x = a.q_up + r * a.ld_up + static_cast<int>(rh % a.H) * (a.dim + a.rot_dim);
    float v = 0.0f;
    if (c < a.dim) {
      v = x[c];
    } else if (c >= dp && c < dp + a.rot_dim) {
      const int p = c - dp, k = p < half ? p : p - half;
      const float2 cs = a.table[(first + r) * half + k];
      const float u = x[a.dim + k], w = x[a.dim + half + k];
      v = p < half ? u * cs.x - w * cs.y : w * cs.x + u * cs.y;
    }
    a.q[i] = from_f<T>(v);
  }
}

// One warp per (query row, head); lanes walk the keys for the scores and the columns for the output.
template <typename T>
__global__ void __launch_bounds__(256) latent_attention_fp32_kernel(const LatentArgs<T> a, int64_t first, int64_t rows) {
  extern __shared__ float qs_all[];   // [8][dim + rot_dim]
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, D = a.dim + a.rot_dim;
  const int dp = (a.dim + 7) / 8 * 8, pitch = latent_q_pitch(a.dim, a.rot_dim);
  float* qs = qs_all + wid * D;
  const int64_t n = rows * a.H;
  for (int64_t it = static_cast<int64_t>(blockIdx.x) * 8 + wid; it < n; it += static_cast<int64_t>(gridDim.x) * 8) {
    const int h = static_cast<int>(it % a.H);
    const int64_t t = it / a.H, r = first + t;
    __syncwarp();
    for (int d = lane; d < D; d += 32) qs[d] = to_f(a.q[it * pitch + (d < a.dim ? d : dp + d - a.dim)]);
    __syncwarp();
    const T* kb = a.kv + h * a.dim;
    const T* vb = a.kv + a.col_v + h * a.vdim;
    float m = -FLT_MAX, l = 0.0f;
    float acc[32];
#pragma unroll
    for (int c = 0; c < 32; ++c) acc[c] = 0.0f;
    for (int64_t jb = 0; jb <= r; jb += 32) {
      const int64_t j = jb + lane;
      float sc = -FLT_MAX;
      if (j <= r) {
        const T* kr = kb + j * a.ld_kv;
        const T* rr = a.cache + j * a.ld_cache + a.rot_col;
        float s0 = 0.0f;
        for (int d = 0; d < a.dim; ++d) s0 = fmaf(qs[d], to_f(kr[d]), s0);
        for (int d = 0; d < a.rot_dim; ++d) s0 = fmaf(qs[a.dim + d], to_f(rr[d]), s0);
        sc = s0 * a.scale;
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
        if (32 * c < a.vdim) {
          float o = acc[c] * c0;
          for (int u = 0; u < nk; ++u) {
            const float pu = __shfl_sync(0xffffffffu, p, u);
            if (d < a.vdim) o = fmaf(pu, to_f(vb[(jb + u) * a.ld_kv + d]), o);
          }
          acc[c] = o;
        }
      }
    }
    const float f = sigmoid_f(a.proj[t * a.ldp + a.col_g + h]) / l;
#pragma unroll
    for (int c = 0; c < 32; ++c) {
      const int d = lane + 32 * c;
      if (d < a.vdim) a.out[t * a.ld_out + h * a.vdim + d] = from_f<T>(acc[c] * f);
    }
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
int latent_prep(const LatentArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s) {
  const int wide = a.q_rank > a.kv_rank ? a.q_rank : a.kv_rank;
  if (a.q_rank % 4 == 0 && a.kv_rank % 4 == 0 && wide <= 1024) {
    const int grid = row_grid(2 * rows, 8);
    if (wide <= 256) LAUNCH("latent prep", (latent_prep4_kernel<T, 2>), grid, 0, a, first, rows);
    if (wide <= 512) LAUNCH("latent prep", (latent_prep4_kernel<T, 4>), grid, 0, a, first, rows);
    LAUNCH("latent prep", (latent_prep4_kernel<T, 8>), grid, 0, a, first, rows);
  }
  LAUNCH("latent prep", latent_prep_kernel<T>, row_grid(2 * rows, 8), 0, a, first, rows);
}
template <typename T>
int latent_rotate(const LatentArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s) {
  if (a.dim % 8 == 0 && a.rot_dim % 16 == 0) LAUNCH("latent rotate", latent_rotate8_kernel<T>, row_grid(rows), 0, a, first, rows);
  LAUNCH("latent rotate", latent_rotate_kernel<T>, row_grid(rows * a.H * latent_q_pitch(a.dim, a.rot_dim), 256), 0, a, first, rows);
}
template <typename T>
int latent_attention_fp32(const LatentArgs<T>& a, int64_t first, int64_t rows, cudaStream_t s) {
  CTDK_REQUIRE(a.vdim <= 1024 && a.dim + a.rot_dim <= 1024, "latent attention: head size above 1024");
  latent_attention_fp32_kernel<T><<<row_grid(rows * a.H, 8), 256, static_cast<size_t>(8) * (a.dim + a.rot_dim) * 4, s>>>(a, first, rows);
  return check_launch("latent attention (fp32)");
}

#define INSTANTIATE(T)                                                                       \
  template int latent_prep<T>(const LatentArgs<T>&, int64_t, int64_t, cudaStream_t);         \
  template int latent_rotate<T>(const LatentArgs<T>&, int64_t, int64_t, cudaStream_t);       \
  template int latent_attention_fp32<T>(const LatentArgs<T>&, int64_t, int64_t, cudaStream_t);
INSTANTIATE(float)
INSTANTIATE(__nv_bfloat16)

}  // namespace hybrid
}  // namespace ctdk
