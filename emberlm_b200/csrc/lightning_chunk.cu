// Lightning attention over long bfloat16 portions, parallel over chunks of 64 tokens:
//   S_t = d S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t   (d per head)
// With S the state in front of a chunk and rows i, j counted inside it:
//   o_i = d^(i+1) S^T q_i + sum_(j <= i) d^(i-j) (q_i . k_j) v_j
//   S'  = d^n S + sum_j d^(n-1-j) k_j v_j^T
// Three kernels: every chunk's own contribution to the state (and silu of q, k, v, kept as bfloat16
// tiles), a scan over the chunks in fp32, and the outputs. q, k, v are bfloat16 (projections with their
// activation); what multiplies them from the recurrence - decayed scores, decayed values, the state -
// is split into a bfloat16 sum of two terms, so the tensor-core products keep 16 mantissa bits of it and
// all sums are fp32. mma.sync m16n8k16, one warp per 16 rows.
#include <cuda_bf16.h>

#include "hybrid_kernels.h"
#include "mma_bf16.cuh"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int C = kLightningChunk;
constexpr int kPad = 8;   // bfloat16 columns behind every shared-memory row: conflict-free ldmatrix

// grid (chunks, heads), 256 threads.
template <int DK, int DV>
__global__ void __launch_bounds__(256, 3) lightning_local_kernel(const LightningArgs a) {
  constexpr int LK = DK + kPad, LV = DV + kPad;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(smem);   // [C][LK]
  __nv_bfloat16* vh = ks + C * LK;                              // [C][LV] high part of the decayed values
  __nv_bfloat16* vl = vh + C * LV;
  __shared__ float pw[C + 1];
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int64_t t0 = static_cast<int64_t>(c) * C;
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);
  if (threadIdx.x <= C) pw[threadIdx.x] = a.powers[h * (C + 1) + threadIdx.x];
  __syncthreads();
  const int64_t tile = static_cast<int64_t>(c) * a.H + h;
  // four columns per thread and turn; head sizes that are not multiples of four load one by one
  const bool vec_k = a.dim % 4 == 0, vec_v = a.vdim % 4 == 0;
  auto fetch = [&](const float* base, int j, int d, int width, bool vec) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j >= n || d >= width) return x;
    const float* p = base + (t0 + j) * a.ldp + h * width + d;
    if (vec) return load4(p);
    x.x = p[0];
    if (d + 1 < width) x.y = p[1];
    if (d + 2 < width) x.z = p[2];
    if (d + 3 < width) x.w = p[3];
    return x;
  };
  auto act = [](const float4& x) { return make_float4(silu_f(x.x), silu_f(x.y), silu_f(x.z), silu_f(x.w)); };
  constexpr int QT = C * DK / 1024, VT = C * DV / 1024;   // turns
#pragma unroll 4
  for (int u = 0; u < QT; ++u) {
    const int i = (threadIdx.x + u * 256) * 4, j = i / DK, d = i % DK;
    const float4 q = act(fetch(a.q, j, d, a.dim, vec_k)), k = act(fetch(a.k, j, d, a.dim, vec_k));
    store4(ks + j * LK + d, k);
    store4(a.kb + tile * (C * DK) + i, k);
    store4(a.qb + tile * (C * DK) + i, q);
  }
#pragma unroll 4
  for (int u = 0; u < VT; ++u) {
    const int i = (threadIdx.x + u * 256) * 4, j = i / DV, d = i % DV;
    const float4 v = act(fetch(a.v, j, d, a.vdim, vec_v));
    __nv_bfloat16* dst = a.vb + tile * (C * DV) + i;
    store4(dst, v);
    const float w = j < n ? pw[n - 1 - j] : 0.0f;
    float s[4] = {v.x, v.y, v.z, v.w}, hi[4], lo[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      s[e] = __bfloat162float(__float2bfloat16(s[e])) * w;   // the stored value, decayed
      hi[e] = __bfloat162float(__float2bfloat16(s[e]));
      lo[e] = s[e] - hi[e];
    }
    store4(vh + j * LV + d, make_float4(hi[0], hi[1], hi[2], hi[3]));
    store4(vl + j * LV + d, make_float4(lo[0], lo[1], lo[2], lo[3]));
  }
  __syncthreads();
  constexpr int MG = DK / 32, NG = 8 / MG, COLS = DV / NG, NT = COLS / 8;
  const int m0 = (wid % MG) * 32, n0 = (wid / MG) * COLS;
  float acc[2][NT][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][t][e] = 0.0f;
#pragma unroll
  for (int k0 = 0; k0 < C; k0 += 16) {
    uint32_t A[2][4];
#pragma unroll
    for (int m = 0; m < 2; ++m) ldsm_a_trans(A[m], ks, LK, m0 + m * 16, k0, lane);
#pragma unroll
    for (int t = 0; t < NT; t += 2) {
      uint32_t B[4];
      ldsm_b_trans(B, vh, LV, k0, n0 + t * 8, lane);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        mma_bf16(acc[m][t], A[m], B[0], B[1]);
        mma_bf16(acc[m][t + 1], A[m], B[2], B[3]);
      }
      ldsm_b_trans(B, vl, LV, k0, n0 + t * 8, lane);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        mma_bf16(acc[m][t], A[m], B[0], B[1]);
        mma_bf16(acc[m][t + 1], A[m], B[2], B[3]);
      }
    }
  }
  float* out = a.chunk_state + tile * (DK * DV);
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      const int r = m0 + m * 16 + (lane >> 2), col = n0 + t * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(out + r * DV + col) = make_float2(acc[m][t][0], acc[m][t][1]);
      *reinterpret_cast<float2*>(out + (r + 8) * DV + col) = make_float2(acc[m][t][2], acc[m][t][3]);
    }
}

// One warp per state row (head, key channel): replaces every chunk's contribution by the state in front
// of the chunk, as two bfloat16 rows (high part, low part) in the same bytes, and stores the last state.
template <int DK, int DV>
__global__ void __launch_bounds__(128) lightning_state_kernel(const LightningArgs a, int chunks) {
  constexpr int N = DV / 32;   // floats per lane
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int h = row / DK, r = row % DK;
  if (h >= a.H) return;
  float S[N];
#pragma unroll
  for (int e = 0; e < N; ++e) {
    const int col = lane * N + e;
    S[e] = (a.resume && r < a.dim && col < a.vdim) ? a.state[(static_cast<int64_t>(h) * a.dim + r) * a.vdim + col] : 0.0f;
  }
  const float* pw = a.powers + h * (C + 1);
  const int64_t step = static_cast<int64_t>(a.H) * DK * DV;
  float* base = a.chunk_state + (static_cast<int64_t>(h) * DK + r) * DV;
  constexpr int U = 4;   // chunks in flight
  for (int c0 = 0; c0 < chunks; c0 += U) {
    float kv[U][N];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int e = 0; e < N; ++e) kv[u][e] = c0 + u < chunks ? __ldcg(base + (c0 + u) * step + lane * N + e) : 0.0f;
    __syncwarp();   // the whole row has been read before any of it is overwritten
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u;
      if (c >= chunks) break;
      __nv_bfloat16* hi = reinterpret_cast<__nv_bfloat16*>(base + c * step);
      const int64_t left = a.rows - static_cast<int64_t>(c) * C;
      const float dn = pw[left < C ? left : C];
      __nv_bfloat16 hh[N], ll[N];
#pragma unroll
      for (int e = 0; e < N; ++e) {
        hh[e] = __float2bfloat16(S[e]);
        ll[e] = __float2bfloat16(S[e] - __bfloat162float(hh[e]));
        S[e] = fmaf(dn, S[e], kv[u][e]);
      }
      if (N == 4) {
        *reinterpret_cast<uint2*>(hi + lane * N) = *reinterpret_cast<uint2*>(hh);
        *reinterpret_cast<uint2*>(hi + DV + lane * N) = *reinterpret_cast<uint2*>(ll);
      } else {
        *reinterpret_cast<uint32_t*>(hi + lane * N) = *reinterpret_cast<uint32_t*>(hh);
        *reinterpret_cast<uint32_t*>(hi + DV + lane * N) = *reinterpret_cast<uint32_t*>(ll);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < N; ++e) {
    const int col = lane * N + e;
    if (r < a.dim && col < a.vdim) a.state[(static_cast<int64_t>(h) * a.dim + r) * a.vdim + col] = S[e];
  }
}

// grid (chunks, heads, DV / 64), 128 threads: a warp owns 16 rows of the chunk and 64 value columns.
template <int DK, int DV>
__global__ void __launch_bounds__(128) lightning_out_kernel(const LightningArgs a) {
  constexpr int LK = DK + kPad, NB = 64, LB = NB + kPad;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem);   // [C][LK]
  __nv_bfloat16* ks = qs + C * LK;                              // [C][LK]
  __nv_bfloat16* vs = ks + C * LK;                              // [C][LB]
  __nv_bfloat16* sh = vs + C * LB;                              // [DK][LB]
  __nv_bfloat16* sl = sh + DK * LB;
  __shared__ float pw[C + 1];
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, n0 = blockIdx.z * NB, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int64_t t0 = static_cast<int64_t>(c) * C, tile = static_cast<int64_t>(c) * a.H + h;
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);
  auto copy = [&](__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, int64_t lds, int rows, int cols) {
    const int per = cols / 8;
    for (int i = threadIdx.x; i < rows * per; i += 128) {
      const int r = i / per, p = i % per;
      cp_async16(dst + r * ld + p * 8, src + r * lds + p * 8);
    }
  };
  copy(qs, LK, a.qb + tile * (C * DK), DK, C, DK);
  copy(ks, LK, a.kb + tile * (C * DK), DK, C, DK);
  copy(vs, LB, a.vb + tile * (C * DV) + n0, DV, C, NB);
  const __nv_bfloat16* st = reinterpret_cast<const __nv_bfloat16*>(a.chunk_state + tile * (DK * DV));
  copy(sh, LB, st + n0, 2 * DV, DK, NB);
  copy(sl, LB, st + DV + n0, 2 * DV, DK, NB);
  cp_async_commit();
  if (threadIdx.x <= C) pw[threadIdx.x] = a.powers[h * (C + 1) + threadIdx.x];
  cp_async_wait_all();
  __syncthreads();
  const int m0 = wid * 16, r0 = m0 + (lane >> 2);
  float sc[8][4], o[8][4];
#pragma unroll
  for (int t = 0; t < 8; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) sc[t][e] = o[t][e] = 0.0f;
#pragma unroll 4
  for (int k0 = 0; k0 < DK; k0 += 16) {
    uint32_t A[4], B[4];
    ldsm_a(A, qs, LK, m0, k0, lane);
#pragma unroll
    for (int t = 0; t < 8; t += 2) {
      if (t * 8 < m0 + 16) {   // keys after the warp's last row are masked anyway
        ldsm_b(B, ks, LK, k0, t * 8, lane);
        mma_bf16(sc[t], A, B[0], B[1]);
        mma_bf16(sc[t + 1], A, B[2], B[3]);
      }
      ldsm_b_trans(B, sh, LB, k0, t * 8, lane);
      mma_bf16(o[t], A, B[0], B[1]);
      mma_bf16(o[t + 1], A, B[2], B[3]);
      ldsm_b_trans(B, sl, LB, k0, t * 8, lane);
      mma_bf16(o[t], A, B[0], B[1]);
      mma_bf16(o[t + 1], A, B[2], B[3]);
    }
  }
  const float d0 = pw[r0 + 1], d1 = pw[r0 + 9];
#pragma unroll
  for (int t = 0; t < 8; ++t) {
    o[t][0] *= d0;
    o[t][1] *= d0;
    o[t][2] *= d1;
    o[t][3] *= d1;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = r0 + (e >> 1) * 8, j = t * 8 + (lane & 3) * 2 + (e & 1);
      sc[t][e] = j <= i ? sc[t][e] * pw[i - j] : 0.0f;
    }
  }
#pragma unroll
  for (int kk = 0; kk < C / 16; ++kk) {
    if (kk * 16 >= m0 + 16) break;
    uint32_t H[4], L[4], B[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float x = sc[2 * kk + (e >> 1)][(e & 1) * 2], y = sc[2 * kk + (e >> 1)][(e & 1) * 2 + 1];
      split_bf16x2(x, y, H[e], L[e]);
    }
#pragma unroll
    for (int t = 0; t < 8; t += 2) {
      ldsm_b_trans(B, vs, LB, kk * 16, t * 8, lane);
      mma_bf16(o[t], H, B[0], B[1]);
      mma_bf16(o[t + 1], H, B[2], B[3]);
      mma_bf16(o[t], L, B[0], B[1]);
      mma_bf16(o[t + 1], L, B[2], B[3]);
    }
  }
  const int64_t ldo = static_cast<int64_t>(a.H) * a.vdim;
  float* out = a.out + t0 * ldo + h * a.vdim;
#pragma unroll
  for (int t = 0; t < 8; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = r0 + (e >> 1) * 8, col = n0 + t * 8 + (lane & 3) * 2 + (e & 1);
      if (i < n && col < a.vdim) out[i * ldo + col] = o[t][e];
    }
}

template <int DK, int DV>
int launch(const LightningArgs& a, cudaStream_t s) {
  const int chunks = static_cast<int>((a.rows + C - 1) / C);
  constexpr size_t m1 = C * (DK + kPad + 2 * (DV + kPad)) * 2;
  constexpr size_t m3 = (2 * C * (DK + kPad) + (C + 2 * DK) * (64 + kPad)) * 2;
  cudaError_t e = cudaFuncSetAttribute(lightning_local_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m1));
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(lightning_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m3));
  if (e == cudaSuccess) e = launch_pdl(lightning_local_kernel<DK, DV>, dim3(chunks, a.H), dim3(256), m1, s, a);
  if (e == cudaSuccess) e = launch_pdl(lightning_state_kernel<DK, DV>, dim3((a.H * DK + 3) / 4), dim3(128), 0, s, a, chunks);
  if (e == cudaSuccess) e = launch_pdl(lightning_out_kernel<DK, DV>, dim3(chunks, a.H, DV / 64), dim3(128), m3, s, a);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "lightning chunks: %s", cudaGetErrorString(e));
  check_launch("lightning chunks");
  check_launch("lightning chunks");
  return check_launch("lightning chunks");
}

}  // namespace

bool lightning_chunked_ok(int dim, int vdim) { return dim <= 128 && vdim <= 128; }

int lightning_chunked(const LightningArgs& a, cudaStream_t s) {
  CTDK_REQUIRE(lightning_chunked_ok(a.dim, a.vdim) && a.H <= 65535, "lightning chunks: head sizes above 128");
  const int dk = lightning_tile(a.dim), dv = lightning_tile(a.vdim);
  if (dk == 64) return dv == 64 ? launch<64, 64>(a, s) : launch<64, 128>(a, s);
  return dv == 64 ? launch<128, 64>(a, s) : launch<128, 128>(a, s);
}

}  // namespace hybrid
}  // namespace ctdk
