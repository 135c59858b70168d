// Mixture of experts over a prompt's portion: routing, the slots of every expert (padded to whole tiles of
// the grouped product), gathering of the rows, and the weighted sum. An expert's rows may stand in any
// order: every row is computed by itself.
#include "decode_core.h"
#include "hybrid_kernels.h"
#include "moe_route.cuh"
#include "parallel_kernels.h"

namespace ctdk {

int gemm_bf16_out16(const void* A, int64_t lda, const void* B, int64_t ldb, __nv_bfloat16* C, int64_t ldc, int64_t M, int N, int K, int up_row,
                    const int32_t* tiles, int max_tiles, int64_t n_pitch, int groups, cudaStream_t stream);

namespace hybrid {
namespace {

int row_grid(int64_t rows, int per_cta = 1) {
  const int64_t need = (rows + per_cta - 1) / per_cta, cap = static_cast<int64_t>(sm_count()) * 16;
  return static_cast<int>(need < cap ? need : cap);
}

__global__ void __launch_bounds__(256) moe_clear_kernel(int32_t* count, int n) {
  pdl_launch();
  pdl_wait();
  for (int i = threadIdx.x; i < n; i += 256) count[i] = 0;
}

// One warp per row. A row's place among its expert's rows is counted in shared memory first, so that the
// counters in global memory see one addition per CTA and expert.
__global__ void __launch_bounds__(256) moe_choose_kernel(const MoeArgs a, int64_t rows) {
  extern __shared__ float sm[];
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int per = a.outputs + route_scratch(a.outputs, a.groups);
  float* z = sm + wid * per;
  int32_t* seen = reinterpret_cast<int32_t*>(sm + 8 * per);   // [experts] of this CTA, then where they start
  for (int e = threadIdx.x; e < a.experts; e += 256) seen[e] = 0;
  __syncthreads();
  const int64_t nw = static_cast<int64_t>(gridDim.x) * 8;
  for (int64_t r = static_cast<int64_t>(blockIdx.x) * 8 + wid; r < rows; r += nw) {
    __syncwarp();
    for (int i = lane; i < a.outputs; i += 32) z[i] = a.z[r * a.ldz + i];
    __syncwarp();
    route_token(z, a.correction, a.outputs, a.groups, a.keep, a.top, z + a.outputs, a.index + r * a.top, a.weight + r * a.top);
    if (lane < a.top) {
      const int e = a.index[r * a.top + lane];
      a.slot[r * a.top + lane] = e < a.experts ? atomicAdd(&seen[e], 1) : 0;
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < a.experts; e += 256)
    if (seen[e] > 0) seen[e] = atomicAdd(&a.count[e], seen[e]);
  __syncthreads();
  for (int64_t r = static_cast<int64_t>(blockIdx.x) * 8 + wid; r < rows; r += nw)
    if (lane < a.top) {
      const int e = a.index[r * a.top + lane];
      if (e < a.experts) a.slot[r * a.top + lane] += seen[e];
    }
}

// One CTA: first tile of every expert, the expert of every tile.
__global__ void __launch_bounds__(1024) moe_tiles_kernel(const MoeArgs a) {
  __shared__ int first[1025];
  pdl_launch();
  pdl_wait();
  const int e = threadIdx.x;
  const int mine = e < a.experts ? (a.count[e] + kMoeTile - 1) / kMoeTile : 0;
  first[e + 1] = mine;
  if (e == 0) first[0] = 0;
  __syncthreads();
  for (int d = 1; d < 1024; d <<= 1) {   // running sum
    const int v = e + 1 > d ? first[e + 1 - d] : 0;
    __syncthreads();
    first[e + 1] += v;
    __syncthreads();
  }
  if (e < a.experts) {
    a.count[a.experts + e] = first[e] * kMoeTile;
    for (int t = first[e]; t < first[e + 1] && t < a.max_tiles; ++t) a.tiles[t] = e;
  }
  if (e == 0) {
    const int n = first[1024] < a.max_tiles ? first[1024] : a.max_tiles;
    a.tiles[a.max_tiles] = n;
    a.tiles[a.max_tiles + 1] = n * kMoeTile;
  }
}

// One warp per chosen output: the row goes to its slot.
template <typename T>
__global__ void __launch_bounds__(256) moe_gather_kernel(const MoeArgs a, const T* __restrict__ h, int64_t ld_h, T* __restrict__ xe, int width,
                                                         int64_t n) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t nw = static_cast<int64_t>(gridDim.x) * 8;
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5; i < n; i += nw) {
    const int e = a.index[i];
    const int slot = e < a.experts ? a.count[a.experts + e] + a.slot[i] : -1;
    __syncwarp();   // every lane has read the place before it becomes the slot
    if (lane == 0) a.slot[i] = slot;
    if (slot < 0) continue;
    const T* src = h + i / a.top * ld_h;
    T* dst = xe + static_cast<int64_t>(slot) * ld_h;
    const int vecs = static_cast<int>(ld_h * sizeof(T) / 16);   // the pitch is a multiple of 8 elements
    constexpr int U = 8;   // in flight
    for (int c0 = lane; c0 < vecs; c0 += 32 * U) {
      uint4 v[U];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (c0 + 32 * u < vecs) v[u] = reinterpret_cast<const uint4*>(src)[c0 + 32 * u];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (c0 + 32 * u < vecs) reinterpret_cast<uint4*>(dst)[c0 + 32 * u] = v[u];
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
    moe_combine_kernel(const MoeArgs a, const T* __restrict__ eo, int64_t ld_eo, const T* __restrict__ h, int64_t ld_h, const float* __restrict__ sg,
                       int64_t ld_sg, const float* __restrict__ shared, float* __restrict__ y, int width, int64_t rows) {
  pdl_launch();
  pdl_wait();
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    const float gate = shared != nullptr ? sigmoid_f(sg[r * ld_sg]) : 0.0f;
    for (int c = threadIdx.x; c < width; c += 256) {
      float v = shared != nullptr ? gate * shared[r * width + c] : 0.0f;
      for (int k = 0; k < a.top; ++k) {
        const int slot = a.slot[r * a.top + k];
        const float u = to_f(slot < 0 ? h[r * ld_h + c] : eo[static_cast<int64_t>(slot) * ld_eo + c]);
        v = fmaf(a.weight[r * a.top + k], u, v);
      }
      y[r * width + c] = v;
    }
  }
}
template <typename T>
__global__ void __launch_bounds__(256)
    moe_combine4_kernel(const MoeArgs a, const T* __restrict__ eo, int64_t ld_eo, const T* __restrict__ h, int64_t ld_h, const float* __restrict__ sg,
                        int64_t ld_sg, const float* __restrict__ shared, float* __restrict__ y, int width, int64_t rows) {
  pdl_launch();
  pdl_wait();
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x) {
    const float gate = shared != nullptr ? sigmoid_f(sg[r * ld_sg]) : 0.0f;
    for (int c = threadIdx.x * 4; c < width; c += 1024) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (shared != nullptr) {
        const float4 u = load4(shared + r * width + c);
        v = make_float4(gate * u.x, gate * u.y, gate * u.z, gate * u.w);
      }
#pragma unroll 4
      for (int k = 0; k < a.top; ++k) {
        const int slot = a.slot[r * a.top + k];
        const float w = a.weight[r * a.top + k];
        const float4 u = load4(slot < 0 ? h + r * ld_h + c : eo + static_cast<int64_t>(slot) * ld_eo + c);
        v = make_float4(fmaf(w, u.x, v.x), fmaf(w, u.y, v.y), fmaf(w, u.z, v.z), fmaf(w, u.w, v.w));
      }
      store4(y + r * width + c, v);
    }
  }
}

// fp32: 64 x 64 output tiles, half a slot tile each, 256 threads with 4 x 4 outputs.
__global__ void __launch_bounds__(256)
    grouped_simt_kernel(const float* __restrict__ A, int64_t lda, const float* __restrict__ W, int64_t ldw, int64_t n_pitch,
                        float* __restrict__ C, int64_t ldc, int N, int K, const int32_t* __restrict__ tiles, int max_tiles) {
  __shared__ float As[16][65], Ws[16][65];
  pdl_launch();
  pdl_wait();
  const int tile = blockIdx.y >> 1;
  if (tile >= tiles[max_tiles]) return;
  const float* w = W + static_cast<int64_t>(tiles[tile]) * n_pitch * ldw;
  const int64_t m0 = static_cast<int64_t>(blockIdx.y) * 64;
  const int n0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = threadIdx.x; i < 1024; i += 256) {
      const int kk = i & 15, mm = i >> 4;
      As[kk][mm] = k0 + kk < K ? A[(m0 + mm) * lda + k0 + kk] : 0.0f;
      Ws[kk][mm] = (n0 + mm < N && k0 + kk < K) ? w[static_cast<int64_t>(n0 + mm) * ldw + k0 + kk] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      float x[4], z[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        x[i] = As[kk][ty * 4 + i];
        z[i] = Ws[kk][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], z[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tx * 4 + j;
      if (c < N) C[(m0 + ty * 4 + i) * ldc + c] = acc[i][j];
    }
}

#define TRY_LAUNCH(what, kernel, grid, block, smem, ...)                                                         \
  do {                                                                                                           \
    const cudaError_t e_ = launch_pdl(kernel, dim3 grid, dim3(block), smem, s, __VA_ARGS__);                     \
    if (e_ != cudaSuccess) return fail(CTDK_ELAUNCH, what ": %s", cudaGetErrorString(e_));                       \
    const int rc_ = check_launch(what);                                                                          \
    if (rc_ != CTDK_OK) return rc_;                                                                              \
  } while (0)

int grouped_simt(const MoeArgs& a, const float* A, int64_t lda, const float* W, int64_t ldw, int64_t n_pitch, float* C, int64_t ldc, int N,
                 int K, cudaStream_t s) {
  TRY_LAUNCH("grouped product (fp32)", grouped_simt_kernel, (static_cast<unsigned>((N + 63) / 64), static_cast<unsigned>(2 * a.max_tiles)), 256,
             0, A, lda, W, ldw, n_pitch, C, ldc, N, K, a.tiles, a.max_tiles);
  return CTDK_OK;
}

}  // namespace

int moe_route(const MoeArgs& a, int64_t rows, cudaStream_t s) {
  CTDK_REQUIRE(a.outputs <= 1024 && a.top <= 32 && a.outputs % a.groups == 0, "moe: more than 1024 outputs or 32 choices");
  TRY_LAUNCH("moe clear", moe_clear_kernel, (1), 256, 0, a.count, 2 * a.experts);
  const size_t smem = (static_cast<size_t>(8) * (a.outputs + route_scratch(a.outputs, a.groups)) + a.experts) * 4;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(moe_choose_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "moe: %s", cudaGetErrorString(e));
  }
  const int64_t ctas = (rows + 7) / 8;
  TRY_LAUNCH("moe choose", moe_choose_kernel, (static_cast<unsigned>(ctas < sm_count() ? ctas : sm_count())), 256, smem, a, rows);
  TRY_LAUNCH("moe tiles", moe_tiles_kernel, (1), 1024, 0, a);
  return CTDK_OK;
}
template <typename T>
int moe_gather(const MoeArgs& a, const T* h, int64_t ld_h, T* xe, int width, int64_t rows, cudaStream_t s) {
  TRY_LAUNCH("moe gather", moe_gather_kernel<T>, (row_grid(rows * a.top, 8)), 256, 0, a, h, ld_h, xe, width, rows * a.top);
  return CTDK_OK;
}
template <typename T>
int moe_combine(const MoeArgs& a, const T* expert_out, int64_t ld_eo, const T* h, int64_t ld_h, const float* sg, int64_t ld_sg, const float* shared,
                float* y, int width, int64_t rows, cudaStream_t s) {
  auto* kernel = width % 4 == 0 ? moe_combine4_kernel<T> : moe_combine_kernel<T>;
  TRY_LAUNCH("moe combine", kernel, (row_grid(rows)), 256, 0, a, expert_out, ld_eo, h, ld_h, sg, ld_sg, shared, y, width, rows);
  return CTDK_OK;
}
int experts_up(const MoeArgs& a, const float* xe, int64_t ld_x, const float* w, int64_t ldw, int K, int effp, float* act, float* scratch,
               cudaStream_t s) {
  DTRY(grouped_simt(a, xe, ld_x, w, ldw, 2 * effp, scratch, 2 * effp, 2 * effp, K, s));
  return glu_rows(scratch, 2 * effp, act, effp, static_cast<int64_t>(a.max_tiles) * kMoeTile, effp, Glu::kSilu, a.tiles + a.max_tiles + 1, s);
}
int experts_up(const MoeArgs& a, const __nv_bfloat16* xe, int64_t ld_x, const __nv_bfloat16* w, int64_t ldw, int K, int effp,
               __nv_bfloat16* act, float*, cudaStream_t s) {
  return gemm_bf16_out16(xe, ld_x, w, ldw, act, effp, static_cast<int64_t>(a.max_tiles) * kMoeTile, effp, K, effp, a.tiles, a.max_tiles,
                         2 * effp, a.experts, s);
}
int experts_down(const MoeArgs& a, const float* act, int64_t ld_a, const float* w, int64_t ldw, int64_t n_pitch, int N, int K, float* out,
                 int64_t ld_out, cudaStream_t s) {
  return grouped_simt(a, act, ld_a, w, ldw, n_pitch, out, ld_out, N, K, s);
}
int experts_down(const MoeArgs& a, const __nv_bfloat16* act, int64_t ld_a, const __nv_bfloat16* w, int64_t ldw, int64_t n_pitch, int N, int K,
                 __nv_bfloat16* out, int64_t ld_out, cudaStream_t s) {
  return gemm_bf16_out16(act, ld_a, w, ldw, out, ld_out, static_cast<int64_t>(a.max_tiles) * kMoeTile, N, K, 0, a.tiles, a.max_tiles, n_pitch,
                         a.experts, s);
}

#define INSTANTIATE(T)                                                                                                            \
  template int moe_gather<T>(const MoeArgs&, const T*, int64_t, T*, int, int64_t, cudaStream_t);                                  \
  template int moe_combine<T>(const MoeArgs&, const T*, int64_t, const T*, int64_t, const float*, int64_t, const float*, float*, int, \
                              int64_t, cudaStream_t);
INSTANTIATE(float)
INSTANTIATE(__nv_bfloat16)

}  // namespace hybrid
}  // namespace ctdk
