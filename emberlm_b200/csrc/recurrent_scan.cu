// Linear-attention recurrences token by token, state in registers (fp32 arithmetic throughout):
//   lightning      S <- decay_h S + k v^T;                         o = S^T q
//   channel delta  S <- diag(e^logg) S; u = beta (v - S^T k); S <- S + k u^T;  o = S^T q
//   wkv            o = (S + diag(bonus) k v^T)^T q;  S <- diag(e^(-e^(z + w0))) S + k v^T
// One CTA owns 32 value columns of a head, one warp four of them; a lane holds every 32nd key row of
// the warp's columns, so a token costs two warp reductions and no block barrier. Inputs are staged 16
// tokens at a time. Used for fp32 models and for short portions; long bfloat16 prompts take the
// chunk-parallel kernels.
#include "hybrid_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int kMaxTile = 16;   // tokens staged at once (half of it for wide keys: 48 KB of static shared memory)

// Sums four values over the warp; lanes 8 j .. 8 j + 7 end up with the sum of value j.
__device__ __forceinline__ float warp_sum4(const float (&v)[4]) {
  const int lane = threadIdx.x & 31;
  const bool hi = (lane & 16) != 0;
  float a0 = hi ? v[2] : v[0], a1 = hi ? v[3] : v[1];
  const float b0 = hi ? v[0] : v[2], b1 = hi ? v[1] : v[3];
  a0 += __shfl_xor_sync(0xffffffffu, b0, 16);
  a1 += __shfl_xor_sync(0xffffffffu, b1, 16);
  const bool odd = (lane & 8) != 0;
  float r = odd ? a1 : a0;
  r += __shfl_xor_sync(0xffffffffu, odd ? a0 : a1, 8);
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
  return r;
}

template <int RPL, Recurrence KIND>
__global__ void __launch_bounds__(256) recurrent_scan_kernel(const ScanArgs a) {
  constexpr bool DELTA = KIND == Recurrence::kDelta, WKV = KIND == Recurrence::kWkv, GATED = DELTA || WKV;
  constexpr int DK = 32 * RPL, kTile = RPL > 4 ? kMaxTile / 2 : kMaxTile;
  __shared__ float q_s[kTile][DK], k_s[kTile][DK], g_s[GATED ? kTile : 1][GATED ? DK : 1], v_s[kTile][32], b_s[kTile];
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int h = blockIdx.y, grp = h / (a.H / a.G), c0 = blockIdx.x * 32;
  const int cw = c0 + wid * 4;   // the warp's first column
  float S[RPL][4];
  float* st = a.state + static_cast<int64_t>(h) * a.dim * a.vdim;
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = lane + 32 * i;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      S[i][j] = (a.resume && r < a.dim && cw + j < a.vdim) ? st[static_cast<int64_t>(r) * a.vdim + cw + j] : 0.0f;
  }
  const float dec = GATED ? 1.0f : a.decay[h];
  float bonus[RPL];
#pragma unroll
  for (int i = 0; i < RPL; ++i) bonus[i] = WKV && lane + 32 * i < a.dim ? a.bonus[h * a.dim + lane + 32 * i] : 0.0f;
  for (int64_t t0 = 0; t0 < a.rows; t0 += kTile) {
    const int nt = static_cast<int>(a.rows - t0 < kTile ? a.rows - t0 : kTile);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * DK; i += 256) {
      const int t = i / DK, d = i % DK;
      float q = 0.0f, k = 0.0f, g = 1.0f;
      if (d < a.dim) {
        q = a.q[(t0 + t) * a.ldq + grp * a.dim + d];
        k = a.k[(t0 + t) * a.ldk + grp * a.dim + d];
        if (a.silu) {
          q = silu_f(q);
          k = silu_f(k);
        }
        if (DELTA) g = expf(a.logg[((t0 + t) * a.H + h) * a.dim + d]);
        if (WKV) g = expf(-expf(a.z[(t0 + t) * a.ldz + h * a.dim + d] + a.w0[h * a.dim + d]));
      }
      q_s[t][d] = q;
      k_s[t][d] = k;
      if (GATED) g_s[t][d] = g;
    }
    for (int i = threadIdx.x; i < nt * 32; i += 256) {
      const int t = i >> 5, c = c0 + (i & 31);
      float v = c < a.vdim ? a.v[(t0 + t) * a.ldv + h * a.vdim + c] : 0.0f;
      if (a.silu) v = silu_f(v);
      v_s[t][i & 31] = v;
    }
    if (DELTA && threadIdx.x < nt) b_s[threadIdx.x] = a.beta[(t0 + threadIdx.x) * a.H + h];
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      float u[4];
      if (DELTA) {
        float p[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
          const float g = g_s[t][lane + 32 * i], k = k_s[t][lane + 32 * i];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            S[i][j] *= g;
            p[j] = fmaf(S[i][j], k, p[j]);
          }
        }
        const float mine = warp_sum4(p);
#pragma unroll
        for (int j = 0; j < 4; ++j) u[j] = b_s[t] * (v_s[t][wid * 4 + j] - __shfl_sync(0xffffffffu, mine, 8 * j));
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) u[j] = v_s[t][wid * 4 + j];
      }
      float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int i = 0; i < RPL; ++i) {
        const float k = k_s[t][lane + 32 * i], q = q_s[t][lane + 32 * i];
        const float keep = WKV ? g_s[WKV ? t : 0][WKV ? lane + 32 * i : 0] : dec;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float kv = k * u[j];
          if (WKV) o[j] = fmaf(fmaf(bonus[i], kv, S[i][j]), q, o[j]);
          S[i][j] = DELTA ? fmaf(k, u[j], S[i][j]) : fmaf(keep, S[i][j], kv);
          if (!WKV) o[j] = fmaf(S[i][j], q, o[j]);
        }
      }
      const float r = warp_sum4(o);
      const int j = lane >> 3;
      if ((lane & 7) == 0 && cw + j < a.vdim) a.out[(t0 + t) * a.H * a.vdim + h * a.vdim + cw + j] = r;
    }
  }
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = lane + 32 * i;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (r < a.dim && cw + j < a.vdim) st[static_cast<int64_t>(r) * a.vdim + cw + j] = S[i][j];
  }
}

template <int RPL>
int launch_scan(const ScanArgs& a, Recurrence kind, cudaStream_t s) {
  const dim3 grid((a.vdim + 31) / 32, a.H);
  auto* kernel = kind == Recurrence::kDelta ? recurrent_scan_kernel<RPL, Recurrence::kDelta>
                 : kind == Recurrence::kWkv ? recurrent_scan_kernel<RPL, Recurrence::kWkv>
                                            : recurrent_scan_kernel<RPL, Recurrence::kLightning>;
  const cudaError_t e = launch_pdl(kernel, grid, dim3(256), 0, s, a);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "recurrent scan: %s", cudaGetErrorString(e));
  return check_launch("recurrent scan");
}

}  // namespace

int recurrent_scan(const ScanArgs& a, Recurrence kind, cudaStream_t s) {
  CTDK_REQUIRE(a.dim >= 1 && a.dim <= 256 && a.H <= 65535, "recurrent scan: key size must be at most 256");
  if (a.dim <= 32) return launch_scan<1>(a, kind, s);
  if (a.dim <= 64) return launch_scan<2>(a, kind, s);
  if (a.dim <= 96) return launch_scan<3>(a, kind, s);
  if (a.dim <= 128) return launch_scan<4>(a, kind, s);
  return launch_scan<8>(a, kind, s);
}

}  // namespace hybrid
}  // namespace ctdk
