// Time mixing with a bonus over long bfloat16 portions, parallel over chunks of 64 tokens:
//   o_t = (S + diag(u) k_t v_t^T)^T r_t,  S <- diag(w_t) S + k_t v_t^T   (w per head and key channel)
// Inside a chunk let b_i be the running sum of the log decays (per channel, inclusive, b_(-1) = 0) and S the
// state in front of it:
//   o_i = (r_i e^(b_(i-1)))^T S + sum_(j < i) (r_i . k_j e^(b_(i-1) - b_j)) v_j + (r_i . u k_i) v_i
//   S'  = diag(e^(b_last)) S + sum_j (k_j e^(b_last - b_j)) v_j^T
// Three kernels: every chunk's own contribution to the state, a scan over the chunks in fp32, and the
// outputs with the norm over each head and the output gate. The pair factors e^(b_(i-1) - b_j) are split:
// between the chunk's halves at the running sum of the boundary, inside a half at that of its middle row,
// provided that no 16 rows decay by more than 2^-kReach in any channel (then both factors stay within fp32
// and bfloat16 range). Otherwise no exponent is ever positive: between 16-row blocks both factors are taken
// relative to the running sum in front of the later block, inside a block the difference is formed per pair.
// r, k, v are bfloat16 (projections); whatever carries a decay is split into
// a bfloat16 sum of two terms before it meets a tensor core (16 mantissa bits, fp32 sums), the state itself
// is carried in fp32. mma.sync m16n8k16.
#include <cuda_bf16.h>

#include "hybrid_kernels.h"
#include "mma_bf16.cuh"
#include "parallel_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int C = kWkvChunk;
constexpr int kPad = 8;        // bfloat16 columns behind every shared-memory row: conflict-free ldmatrix
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kFloor = -150.0f;   // a log2 decay below this wipes the channel either way
constexpr float kReach = 100.0f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Four columns from p, `left` of them existing.
__device__ __forceinline__ float4 fetch4(const float* p, int left, bool vec) {
  float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
  if (left <= 0) return x;
  if (vec) return load4(p);
  x.x = p[0];
  if (left > 1) x.y = p[1];
  if (left > 2) x.z = p[2];
  if (left > 3) x.w = p[3];
  return x;
}
__device__ __forceinline__ float log2_decay(float z) { return fmaxf(-ex2(z * kLog2e) * kLog2e, kFloor); }
__device__ __forceinline__ void put_split(__nv_bfloat16* hi, __nv_bfloat16* lo, const float4& v) {
  uint32_t h0, l0, h1, l1;
  split_bf16x2(v.x, v.y, h0, l0);
  split_bf16x2(v.z, v.w, h1, l1);
  *reinterpret_cast<uint2*>(hi) = make_uint2(h0, h1);
  *reinterpret_cast<uint2*>(lo) = make_uint2(l0, l1);
}

// b_s [C][LB]: log decays in, running sums over the rows out; scratch of 256 floats. 256 threads.
template <int D, int LB>
__device__ __forceinline__ void running_sums(float* b_s, float* scratch) {
  constexpr int SEG = 256 / D, ROWS = C / SEG;
  const int d = threadIdx.x % D, sg = threadIdx.x / D;
  float s = 0.0f;
#pragma unroll 8
  for (int r = 0; r < ROWS; ++r) s += b_s[(sg * ROWS + r) * LB + d];
  scratch[sg * D + d] = s;
  __syncthreads();
  float run = 0.0f;
  for (int e = 0; e < sg; ++e) run += scratch[e * D + d];
#pragma unroll 8
  for (int r = 0; r < ROWS; ++r) {
    float* p = b_s + (sg * ROWS + r) * LB + d;
    run += *p;
    *p = run;
  }
  __syncthreads();
}

template <int D>
struct LocalCfg {
  static constexpr int LB = D + 4, L = D + kPad;
  static constexpr int kBytes = C * LB * 4 + 256 * 4 + 3 * C * L * 2;
};

// grid (chunks, heads), 256 threads: chunk_state = K_decayed^T V, decay = e^(b_last).
template <int D>
__global__ void __launch_bounds__(256) wkv_local_kernel(const WkvArgs a) {
  using Cfg = LocalCfg<D>;
  constexpr int LB = Cfg::LB, L = Cfg::L, T = C * D / 1024;
  extern __shared__ __align__(16) unsigned char smem[];
  float* b_s = reinterpret_cast<float*>(smem);
  float* scratch = b_s + C * LB;
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(scratch + 256);   // [C][L]
  __nv_bfloat16* kl = kh + C * L;
  __nv_bfloat16* vs = kl + C * L;
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int64_t t0 = static_cast<int64_t>(c) * C, tile = static_cast<int64_t>(c) * a.H + h;
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);
  const bool vec = a.dim % 4 == 0;
  float4 k[T];
#pragma unroll
  for (int u = 0; u < T; ++u) {
    const int i = (threadIdx.x + u * 256) * 4, r = i / D, d = i % D, left = r < n ? a.dim - d : 0;
    const int64_t at = (t0 + r) * a.ldp + h * a.dim + d;
    k[u] = fetch4(a.k + at, left, vec);
    const float4 v = fetch4(a.v + at, left, vec);
    const float4 z = fetch4(a.z + (t0 + r) * a.ldz + h * a.dim + d, left, vec), w = fetch4(a.w0 + h * a.dim + d, left, vec);
    store4(vs + r * L + d, v);
    float4 g = make_float4(0.f, 0.f, 0.f, 0.f);
    if (left > 0) g = make_float4(log2_decay(z.x + w.x), log2_decay(z.y + w.y), log2_decay(z.z + w.z), log2_decay(z.w + w.w));
    store4(b_s + r * LB + d, g);
  }
  __syncthreads();
  running_sums<D, LB>(b_s, scratch);
#pragma unroll
  for (int u = 0; u < T; ++u) {
    const int i = (threadIdx.x + u * 256) * 4, r = i / D, d = i % D;
    const float4 b = load4(b_s + r * LB + d), e = load4(b_s + (C - 1) * LB + d);
    auto q = [](float x) { return __bfloat162float(__float2bfloat16(x)); };
    put_split(kh + r * L + d, kl + r * L + d,
              make_float4(q(k[u].x) * ex2(e.x - b.x), q(k[u].y) * ex2(e.y - b.y), q(k[u].z) * ex2(e.z - b.z), q(k[u].w) * ex2(e.w - b.w)));
    if (r == C - 1) store4(a.decay + tile * D + d, make_float4(ex2(e.x), ex2(e.y), ex2(e.z), ex2(e.w)));
  }
  __syncthreads();
  constexpr int MG = D / 32, NG = 8 / MG, COLS = D / NG, NT = COLS / 8;
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
    uint32_t A[2][4], Al[2][4];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      ldsm_a_trans(A[m], kh, L, m0 + m * 16, k0, lane);
      ldsm_a_trans(Al[m], kl, L, m0 + m * 16, k0, lane);
    }
#pragma unroll
    for (int t = 0; t < NT; t += 2) {
      uint32_t B[4];
      ldsm_b_trans(B, vs, L, k0, n0 + t * 8, lane);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        mma_bf16(acc[m][t], A[m], B[0], B[1]);
        mma_bf16(acc[m][t + 1], A[m], B[2], B[3]);
        mma_bf16(acc[m][t], Al[m], B[0], B[1]);
        mma_bf16(acc[m][t + 1], Al[m], B[2], B[3]);
      }
    }
  }
  float* out = a.chunk_state + tile * (D * D);
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      const int r = m0 + m * 16 + (lane >> 2), col = n0 + t * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(out + r * D + col) = make_float2(acc[m][t][0], acc[m][t][1]);
      *reinterpret_cast<float2*>(out + (r + 8) * D + col) = make_float2(acc[m][t][2], acc[m][t][3]);
    }
}

// One warp per state row (head, key channel): replaces every chunk's contribution by the state in front of
// the chunk, as two bfloat16 rows (high part, low part) in the same bytes, and stores the last state.
template <int D>
__global__ void __launch_bounds__(128) wkv_state_kernel(const WkvArgs a, int chunks) {
  constexpr int N = D / 32, U = 8;   // floats per lane, chunks in flight
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, row = blockIdx.x * 4 + (threadIdx.x >> 5), h = row / D, r = row % D;
  if (h >= a.H) return;
  float S[N];
#pragma unroll
  for (int e = 0; e < N; ++e) {
    const int col = lane * N + e;
    S[e] = (a.resume && r < a.dim && col < a.dim) ? a.state[(static_cast<int64_t>(h) * a.dim + r) * a.dim + col] : 0.0f;
  }
  const int64_t step = static_cast<int64_t>(a.H) * D * D;
  float* base = a.chunk_state + (static_cast<int64_t>(h) * D + r) * D;
  const float* decay = a.decay + static_cast<int64_t>(h) * D + r;
  for (int c0 = 0; c0 < chunks; c0 += U) {
    float kv[U][N], dec[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      dec[u] = c0 + u < chunks ? __ldcg(decay + static_cast<int64_t>(c0 + u) * a.H * D) : 0.0f;
#pragma unroll
      for (int e = 0; e < N; ++e) kv[u][e] = c0 + u < chunks ? __ldcg(base + (c0 + u) * step + lane * N + e) : 0.0f;
    }
    __syncwarp();   // the whole row has been read before any of it is overwritten
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u >= chunks) break;
      __nv_bfloat16* hi = reinterpret_cast<__nv_bfloat16*>(base + (c0 + u) * step);
      __nv_bfloat16 hh[N], ll[N];
#pragma unroll
      for (int e = 0; e < N; ++e) {
        hh[e] = __float2bfloat16(S[e]);
        ll[e] = __float2bfloat16(S[e] - __bfloat162float(hh[e]));
        S[e] = fmaf(dec[u], S[e], kv[u][e]);
      }
#pragma unroll
      for (int e = 0; e < N; e += 2) {
        *reinterpret_cast<__nv_bfloat162*>(hi + lane * N + e) = __nv_bfloat162(hh[e], hh[e + 1]);
        *reinterpret_cast<__nv_bfloat162*>(hi + D + lane * N + e) = __nv_bfloat162(ll[e], ll[e + 1]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < N; ++e) {
    const int col = lane * N + e;
    if (r < a.dim && col < a.dim) a.state[(static_cast<int64_t>(h) * a.dim + r) * a.dim + col] = S[e];
  }
}

template <int D>
struct OutCfg {
  static constexpr int LB = D + 4, L = D + kPad, LA = C + kPad;
  // b, r, k, v, (query factors | r e^b) x 2, (key factors | scores) x 2, state x 2
  static_assert(L >= LA, "the scores lie where the key factors were");
  static constexpr int kBytes = C * LB * 4 + 3 * C * L * 2 + 2 * C * L * 2 + 2 * C * L * 2 + 2 * D * L * 2 + 256 * 4 + D * 4;
};

// grid (chunks, heads), 256 threads.
template <int D>
__global__ void __launch_bounds__(256) wkv_out_kernel(const WkvArgs a) {
  using Cfg = OutCfg<D>;
  constexpr int LB = Cfg::LB, L = Cfg::L, LA = Cfg::LA, T = C * D / 1024;
  extern __shared__ __align__(16) unsigned char smem[];
  float* b_s = reinterpret_cast<float*>(smem);                          // [C][LB]
  float* scratch = b_s + C * LB;                                        // [256]
  float* u_s = scratch + 256;                                           // [D]
  __nv_bfloat16* rs = reinterpret_cast<__nv_bfloat16*>(u_s + D);        // [C][L]
  __nv_bfloat16* ks = rs + C * L;
  __nv_bfloat16* vs = ks + C * L;
  __nv_bfloat16* fh = vs + C * L;                                       // [C][L] factors, high and low
  __nv_bfloat16* fl = fh + C * L;
  __nv_bfloat16* ah = fl + C * L;                                       // [C][LA] scores, high and low
  __nv_bfloat16* al = ah + C * L;
  __nv_bfloat16* sh = al + C * L;                                       // [D][L] state, high and low
  __nv_bfloat16* sl = sh + D * L;
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const int64_t t0 = static_cast<int64_t>(c) * C, tile = static_cast<int64_t>(c) * a.H + h;
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);
  const bool vec = a.dim % 4 == 0;
  {
    const __nv_bfloat16* st = reinterpret_cast<const __nv_bfloat16*>(a.chunk_state + tile * (D * D));
    constexpr int P = D / 8;
    for (int i = tid; i < D * P; i += 256) {
      const int r = i / P, p = i % P * 8;
      cp_async16(sh + r * L + p, st + r * 2 * D + p);
      cp_async16(sl + r * L + p, st + r * 2 * D + D + p);
    }
    cp_async_commit();
  }
#pragma unroll
  for (int u = 0; u < T; ++u) {
    const int i = (tid + u * 256) * 4, r = i / D, d = i % D, left = r < n ? a.dim - d : 0;
    const int64_t at = (t0 + r) * a.ldp + h * a.dim + d;
    const float4 q = fetch4(a.r + at, left, vec), k = fetch4(a.k + at, left, vec), v = fetch4(a.v + at, left, vec);
    const float4 z = fetch4(a.z + (t0 + r) * a.ldz + h * a.dim + d, left, vec), w = fetch4(a.w0 + h * a.dim + d, left, vec);
    store4(rs + r * L + d, q);
    store4(ks + r * L + d, k);
    store4(vs + r * L + d, v);
    float4 g = make_float4(0.f, 0.f, 0.f, 0.f);
    if (left > 0) g = make_float4(log2_decay(z.x + w.x), log2_decay(z.y + w.y), log2_decay(z.z + w.z), log2_decay(z.w + w.w));
    store4(b_s + r * LB + d, g);
  }
  for (int d = tid; d < D; d += 256) u_s[d] = d < a.dim ? a.bonus[h * a.dim + d] : 0.0f;
  __syncthreads();
  running_sums<D, LB>(b_s, scratch);

  float reach = 0.0f;
  for (int x = tid; x < 4 * D; x += 256) {
    const int d = x % D, q = x / D;
    reach = fminf(reach, b_s[(16 * q + 15) * LB + d] - (q > 0 ? b_s[(16 * q - 1) * LB + d] : 0.0f));
  }
  if (__syncthreads_or(reach < -kReach) == 0) {
    __nv_bfloat16 *xh = ah, *xl = al;   // [C][L] key factors, where the scores will be
    auto query_factor = [&](int r, int d, const float4& z) {
      const float4 q = load4(rs + r * L + d), p = r > 0 ? load4(b_s + (r - 1) * LB + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      put_split(fh + r * L + d, fl + r * L + d, make_float4(q.x * ex2(p.x - z.x), q.y * ex2(p.y - z.y), q.z * ex2(p.z - z.z), q.w * ex2(p.w - z.w)));
    };
    auto key_factor = [&](int r, int d, const float4& z) {
      const float4 k = load4(ks + r * L + d), b = load4(b_s + r * LB + d);
      put_split(xh + r * L + d, xl + r * L + d, make_float4(k.x * ex2(z.x - b.x), k.y * ex2(z.y - b.y), k.z * ex2(z.z - b.z), k.w * ex2(z.w - b.w)));
    };
    // a warp has 16 rows and 32 columns of the scores; tiles above the diagonal are left out
    const int i0 = (wid & 3) * 16, j0 = (wid >> 2) * 32;
    float acc[4][4] = {};
    auto scores = [&] {
#pragma unroll 2
      for (int k0 = 0; k0 < D; k0 += 16) {
        uint32_t Ah[4], Al[4];
        ldsm_a(Ah, fh, L, i0, k0, lane);
        ldsm_a(Al, fl, L, i0, k0, lane);
#pragma unroll
        for (int t = 0; t < 4; t += 2) {
          if (j0 + t * 8 >= i0 + 16) break;
          uint32_t Bh[4], Bl[4];
          ldsm_b(Bh, xh, L, k0, j0 + t * 8, lane);
          ldsm_b(Bl, xl, L, k0, j0 + t * 8, lane);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mma_bf16(acc[t + e], Ah, Bh[2 * e], Bh[2 * e + 1]);
            mma_bf16(acc[t + e], Ah, Bl[2 * e], Bl[2 * e + 1]);
            mma_bf16(acc[t + e], Al, Bh[2 * e], Bh[2 * e + 1]);
          }
        }
      }
    };
#pragma unroll
    for (int u = 0; u < T; ++u) {   // inside the halves
      const int i = (tid + u * 256) * 4, r = i / D, d = i % D;
      const float4 z = load4(b_s + ((r & 32) + 15) * LB + d);
      query_factor(r, d, z);
      key_factor(r, d, z);
    }
    {   // the bonus terms, four threads per row
      const int i = tid >> 2;
      float s = 0.0f;
#pragma unroll 4
      for (int d = (tid & 3) * 4; d < D; d += 16) {
        const float4 r = load4(rs + i * L + d), k = load4(ks + i * L + d), u = load4(u_s + d);
        s = fmaf(r.x * k.x, u.x, fmaf(r.y * k.y, u.y, fmaf(r.z * k.z, u.z, fmaf(r.w * k.w, u.w, s))));
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      if ((tid & 3) == 0) scratch[i] = s;
    }
    __syncthreads();
    if ((i0 & 32) == j0) scores();
    __syncthreads();
#pragma unroll
    for (int u = 0; u < T / 2; ++u) {   // queries of the second half, keys of the first
      const int i = (tid + u * 256) * 4, r = i / D, d = i % D;
      const float4 z = load4(b_s + 31 * LB + d);
      query_factor(r + 32, d, z);
      key_factor(r, d, z);
    }
    __syncthreads();
    if (i0 >= 32 && j0 == 0) scores();
    __syncthreads();
#pragma unroll
    for (int t = 0; t < 4; ++t)
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int i = i0 + (lane >> 2) + 8 * f, j = j0 + 8 * t + (lane & 3) * 2;
        const float x = j < i ? acc[t][2 * f] : (j == i ? scratch[i] : 0.0f);
        const float y = j + 1 < i ? acc[t][2 * f + 1] : (j + 1 == i ? scratch[i] : 0.0f);
        uint32_t hi, lo;
        split_bf16x2(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(ah + i * LA + j) = hi;
        *reinterpret_cast<uint32_t*>(al + i * LA + j) = lo;
      }
  } else {
    for (int i = tid; i < C * LA / 4; i += 256) reinterpret_cast<uint2*>(ah)[i] = reinterpret_cast<uint2*>(al)[i] = make_uint2(0u, 0u);
    __syncthreads();
    // pairs inside a 16-row block: a thread has row i and the columns jq, jq + 4, ... up to i
    {
      const int blk = tid >> 6 << 4, il = (tid >> 2) & 15, jq = tid & 3, i = blk + il;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      const float* bi = b_s + (i - 1) * LB;
#pragma unroll 2
      for (int d = 0; d < D; d += 4) {
        const float4 r = load4(rs + i * L + d), u = load4(u_s + d);
        const float4 b = i > 0 ? load4(bi + d) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int jl = jq + 4 * e, j = blk + jl;
          if (jl > il) break;
          const float4 k = load4(ks + j * L + d);
          float4 f = u;
          if (jl < il) {
            const float4 bj = load4(b_s + j * LB + d);
            f = make_float4(ex2(b.x - bj.x), ex2(b.y - bj.y), ex2(b.z - bj.z), ex2(b.w - bj.w));
          }
          s[e] = fmaf(r.x * k.x, f.x, fmaf(r.y * k.y, f.y, fmaf(r.z * k.z, f.z, fmaf(r.w * k.w, f.w, s[e]))));
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int jl = jq + 4 * e;
        if (jl > il) break;
        const __nv_bfloat16 hi = __float2bfloat16(s[e]);
        ah[i * LA + blk + jl] = hi;
        al[i * LA + blk + jl] = __float2bfloat16(s[e] - __bfloat162float(hi));
      }
    }
    // pairs in different blocks: rows of block I against all rows before it
    for (int I = 1; I < C / 16; ++I) {
      const float* ref = b_s + (16 * I - 1) * LB;
      for (int x = tid * 4; x < 16 * (I + 1) * D; x += 1024) {
        const int r = x / D, d = x % D;
        const float4 z = load4(ref + d);
        float4 f;
        if (r < 16 * I) {
          const float4 b = load4(b_s + r * LB + d), k = load4(ks + r * L + d);
          f = make_float4(k.x * ex2(z.x - b.x), k.y * ex2(z.y - b.y), k.z * ex2(z.z - b.z), k.w * ex2(z.w - b.w));
        } else {
          const float4 b = load4(b_s + (r - 1) * LB + d), q = load4(rs + r * L + d);
          f = make_float4(q.x * ex2(b.x - z.x), q.y * ex2(b.y - z.y), q.z * ex2(b.z - z.z), q.w * ex2(b.w - z.w));
        }
        put_split(fh + r * L + d, fl + r * L + d, f);
      }
      __syncthreads();
      if (wid < I) {   // a warp per 16 x 16 block of scores
        float acc[2][4] = {};
#pragma unroll 2
        for (int k0 = 0; k0 < D; k0 += 16) {
          uint32_t Ah[4], Al[4], Bh[4], Bl[4];
          ldsm_a(Ah, fh, L, 16 * I, k0, lane);
          ldsm_a(Al, fl, L, 16 * I, k0, lane);
          ldsm_b(Bh, fh, L, k0, 16 * wid, lane);
          ldsm_b(Bl, fl, L, k0, 16 * wid, lane);
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            mma_bf16(acc[t], Ah, Bh[2 * t], Bh[2 * t + 1]);
            mma_bf16(acc[t], Ah, Bl[2 * t], Bl[2 * t + 1]);
            mma_bf16(acc[t], Al, Bh[2 * t], Bh[2 * t + 1]);
          }
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int f = 0; f < 2; ++f) {
            const int i = 16 * I + (lane >> 2) + 8 * f, j = 16 * wid + 8 * t + (lane & 3) * 2;
            uint32_t hi, lo;
            split_bf16x2(acc[t][2 * f], acc[t][2 * f + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(ah + i * LA + j) = hi;
            *reinterpret_cast<uint32_t*>(al + i * LA + j) = lo;
          }
      }
      __syncthreads();
    }
  }
  // r e^(b_(i-1)) takes the factors' place
#pragma unroll
  for (int u = 0; u < T; ++u) {
    const int i = (tid + u * 256) * 4, r = i / D, d = i % D;
    float4 q = load4(rs + r * L + d);
    if (r > 0) {
      const float4 b = load4(b_s + (r - 1) * LB + d);
      q = make_float4(q.x * ex2(b.x), q.y * ex2(b.y), q.z * ex2(b.z), q.w * ex2(b.w));
    }
    put_split(fh + r * L + d, fl + r * L + d, q);
  }
  cp_async_wait_all();
  __syncthreads();
  constexpr int NT = D / 16;   // column tiles of a warp: half of the head
  const int m0 = (wid & 3) * 16, n0 = (wid >> 2) * (D / 2);
  float o[NT][4];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[t][e] = 0.0f;
#pragma unroll 2
  for (int k0 = 0; k0 < D; k0 += 16) {
    uint32_t Ah[4], Al[4];
    ldsm_a(Ah, fh, L, m0, k0, lane);
    ldsm_a(Al, fl, L, m0, k0, lane);
#pragma unroll
    for (int t = 0; t < NT; t += 2) {
      uint32_t Bh[4], Bl[4];
      ldsm_b_trans(Bh, sh, L, k0, n0 + t * 8, lane);
      ldsm_b_trans(Bl, sl, L, k0, n0 + t * 8, lane);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mma_bf16(o[t + e], Ah, Bh[2 * e], Bh[2 * e + 1]);
        mma_bf16(o[t + e], Ah, Bl[2 * e], Bl[2 * e + 1]);
        mma_bf16(o[t + e], Al, Bh[2 * e], Bh[2 * e + 1]);
      }
    }
  }
#pragma unroll
  for (int k0 = 0; k0 < C; k0 += 16) {
    if (k0 >= m0 + 16) break;
    uint32_t Ah[4], Al[4];
    ldsm_a(Ah, ah, LA, m0, k0, lane);
    ldsm_a(Al, al, LA, m0, k0, lane);
#pragma unroll
    for (int t = 0; t < NT; t += 2) {
      uint32_t B[4];
      ldsm_b_trans(B, vs, L, k0, n0 + t * 8, lane);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mma_bf16(o[t + e], Ah, B[2 * e], B[2 * e + 1]);
        mma_bf16(o[t + e], Al, B[2 * e], B[2 * e + 1]);
      }
    }
  }
  // norm over the head (columns past dim are zero), weight, gate
  float ss[2] = {0.0f, 0.0f};
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) ss[e >> 1] = fmaf(o[t][e], o[t][e], ss[e >> 1]);
#pragma unroll
  for (int f = 0; f < 2; ++f) {
    ss[f] += __shfl_xor_sync(0xffffffffu, ss[f], 1);
    ss[f] += __shfl_xor_sync(0xffffffffu, ss[f], 2);
    if ((lane & 3) == 0) scratch[(wid >> 2) * C + m0 + (lane >> 2) + 8 * f] = ss[f];
  }
  __syncthreads();
  const bool pairs = a.dim % 2 == 0;
#pragma unroll
  for (int f = 0; f < 2; ++f) {
    const int i = m0 + (lane >> 2) + 8 * f;
    if (i >= n) continue;
    const float sc = rsqrtf((scratch[i] + scratch[C + i]) / static_cast<float>(a.dim) + a.eps);
    const float* gate = a.gate + (t0 + i) * a.ldp + h * a.dim;
    const float* w = a.w_norm + h * a.dim;
    __nv_bfloat16* dst = a.out + (t0 + i) * a.ld_out + h * a.dim;
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      const int col = n0 + t * 8 + (lane & 3) * 2;
      const float x = o[t][2 * f] * sc, y = o[t][2 * f + 1] * sc;
      if (pairs && col < a.dim) {
        const float2 g = *reinterpret_cast<const float2*>(gate + col), p = *reinterpret_cast<const float2*>(w + col);
        *reinterpret_cast<__nv_bfloat162*>(dst + col) = __floats2bfloat162_rn(x * p.x * silu_f(g.x), y * p.y * silu_f(g.y));
      } else {
        if (col < a.dim) dst[col] = __float2bfloat16(x * w[col] * silu_f(gate[col]));
        if (col + 1 < a.dim) dst[col + 1] = __float2bfloat16(y * w[col + 1] * silu_f(gate[col + 1]));
      }
    }
  }
}

template <int D>
int launch(const WkvArgs& a, cudaStream_t s) {
  const int chunks = static_cast<int>((a.rows + C - 1) / C);
  constexpr int m1 = LocalCfg<D>::kBytes, m3 = OutCfg<D>::kBytes;
  cudaError_t e = cudaFuncSetAttribute(wkv_local_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, m1);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(wkv_out_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, m3);
  if (e == cudaSuccess) e = launch_pdl(wkv_local_kernel<D>, dim3(chunks, a.H), dim3(256), m1, s, a);
  if (e == cudaSuccess) e = launch_pdl(wkv_state_kernel<D>, dim3((a.H * D + 3) / 4), dim3(128), 0, s, a, chunks);
  if (e == cudaSuccess) e = launch_pdl(wkv_out_kernel<D>, dim3(chunks, a.H), dim3(256), m3, s, a);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "wkv chunks: %s", cudaGetErrorString(e));
  check_launch("wkv chunks");
  check_launch("wkv chunks");
  return check_launch("wkv chunks");
}

}  // namespace

bool wkv_chunked_ok(int dim) { return dim <= 128; }

int wkv_chunked(const WkvArgs& a, cudaStream_t s) {
  CTDK_REQUIRE(wkv_chunked_ok(a.dim) && a.H <= 65535, "wkv chunks: head size above 128");
  return wkv_tile(a.dim) == 64 ? launch<64>(a, s) : launch<128>(a, s);
}

}  // namespace hybrid
}  // namespace ctdk
