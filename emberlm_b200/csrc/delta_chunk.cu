// Delta rule with one decay per key channel over long portions, parallel over chunks of 64 tokens. Inside a chunk let b_i be the running sum of the log decays (per channel,
// inclusive) and S the state in front of it. Unrolling
//   S <- diag(g) S;  u_i = beta_i (v_i - S^T k_i);  S <- S + k_i u_i^T;  o_i = S^T q_i
// gives, with A_ij = sum_c k_ic k_jc e^(b_ic - b_jc) (j < i) and B_ij the same with q_i (j <= i),
//   (I + diag(beta) A) U = diag(beta) (V - (K e^b) S)
//   O = (Q e^b) S + B U,      S' = diag(e^(b_last)) S + (K e^(b_last - b))^T U
// so with T = (I + diag(beta) A)^-1 diag(beta): U = T V - (T K e^b) S. Kernels:
//   delta_local  per (chunk, head): b, A, B, the triangular inverse, T V, W = T K e^b
//   delta_state  per (head, 16 value columns): U and S, chunk after chunk
//   delta_out    per (chunk, head): O
// Exponents are differences b_i - b_j with j <= i only, never positive: between 16-row blocks both
// factors are taken relative to the running sum in front of the later block, inside a block the
// difference is formed per pair. Strong decays underflow to zero and nothing overflows.
//
// delta_local is fp32 arithmetic throughout. The other two exist twice: in fp32, and (split, for
// bfloat16 models) on the tensor cores with every factor - W, K e^.., Q e^.., U, B and the fp32 state -
// split into a bfloat16 sum of two terms, x y = xh yh + xh yl + xl yh: 16 mantissa bits of each factor,
// fp32 sums, the state itself kept in fp32. Shared memory feeds an fp32 tile product at half the FMA
// rate at best (a 128-bit load per warp occupies it for four cycles, whatever it broadcasts), which made
// the serial state kernel five times slower than the split form.
#include "hybrid_kernels.h"
#include "mma_bf16.cuh"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int C = kDeltaChunk;
constexpr int LT = C + 4;   // pitch of 64-column tiles
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
  acc = fmaf(a.x, b.x, acc);
  acc = fmaf(a.y, b.y, acc);
  acc = fmaf(a.z, b.z, acc);
  return fmaf(a.w, b.w, acc);
}
__device__ __forceinline__ void axpy4(float s, const float4& b, float (&acc)[4]) {
  acc[0] = fmaf(s, b.x, acc[0]);
  acc[1] = fmaf(s, b.y, acc[1]);
  acc[2] = fmaf(s, b.z, acc[2]);
  acc[3] = fmaf(s, b.w, acc[3]);
}
__device__ __forceinline__ float lane4(const float4& v, int e) { return e == 0 ? v.x : e == 1 ? v.y : e == 2 ? v.z : v.w; }

// acc[4][4] += M[r0 .. r0 + 3][0 .. nk) N[0 .. nk)[c0 .. c0 + 3] (nk a multiple of 4)
__device__ __forceinline__ void tile_product(const float* M, int ldm, const float* N, int ldn, int r0, int c0, int nk, float (&acc)[4][4]) {
#pragma unroll 2
  for (int k = 0; k < nk; k += 4) {
    float4 m[4], x[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      m[e] = ld4(M + (r0 + e) * ldm + k);
      x[e] = ld4(N + (k + e) * ldn + c0);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int e = 0; e < 4; ++e) axpy4(lane4(m[r], e), x[e], acc[r]);
  }
}

// Two bfloat16 planes [2][rows][cols] in the bytes of an fp32 tile.
__device__ __forceinline__ void store_split(float* tile, int plane, int i, const float4& v) {
  __nv_bfloat16* p = reinterpret_cast<__nv_bfloat16*>(tile);
  uint32_t h0, l0, h1, l1;
  split_bf16x2(v.x, v.y, h0, l0);
  split_bf16x2(v.z, v.w, h1, l1);
  *reinterpret_cast<uint2*>(p + i) = make_uint2(h0, h1);
  *reinterpret_cast<uint2*>(p + plane + i) = make_uint2(l0, l1);
}
template <bool SPLIT>
__device__ __forceinline__ void put4(float* tile, int plane, int i, const float4& v) {
  if (SPLIT) store_split(tile, plane, i, v);
  else store4(tile + i, v);
}

template <int DK, int DV>
struct LocalCfg {
  static constexpr int LD = DK + 4, LV = DV + 4;
  static constexpr int kRows = 3 * C * LD > 2 * C * LD + C * LV ? 3 * C * LD : 2 * C * LD + C * LV;   // b, k, then q or v
  static constexpr int kFloats = kRows + 48 * LD + 2 * 16 * LD + 2 * C * LT + 3 * 16 * 17 + C;
};

// grid (chunks, heads), 512 threads.
template <int DK, int DV, bool SPLIT>
__global__ void __launch_bounds__(512, 1) delta_local_kernel(const DeltaChunkArgs a) {
  using Cfg = LocalCfg<DK, DV>;
  constexpr int LD = Cfg::LD, LV = Cfg::LV;
  extern __shared__ __align__(16) float sm[];
  float* b_s = sm;                   // [C][LD] running log2 decay
  float* k_s = b_s + C * LD;         // [C][LD]
  float* q_s = k_s + C * LD;         // [C][LD]; later the values [C][LV]
  float* kx = sm + Cfg::kRows;       // [48][LD] earlier keys relative to a block's start
  float* kr = kx + 48 * LD;          // [16][LD] the block's own keys
  float* qr = kr + 16 * LD;          // [16][LD]
  float* L_s = qr + 16 * LD;         // [C][LT] diag(beta) A, strictly lower
  float* X_s = L_s + C * LT;         // [C][LT] its (I + L)^-1, later T
  float* tmp = X_s + C * LT;         // [3][16][17]
  float* be = tmp + 3 * 16 * 17;     // [C]
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, grp = h / (a.H / a.G), tid = threadIdx.x;
  const int64_t t0 = static_cast<int64_t>(c) * C, tile = static_cast<int64_t>(c) * a.H + h;
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);

  // four columns per thread and turn; head sizes that are not multiples of four load one by one
  auto fetch = [](const float* p, int left, bool vec) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (left <= 0) return x;
    if (vec) return ld4(p);
    x.x = p[0];
    if (left > 1) x.y = p[1];
    if (left > 2) x.z = p[2];
    if (left > 3) x.w = p[3];
    return x;
  };
  const bool vec_k = a.dim % 4 == 0, vec_v = a.vdim % 4 == 0;
  constexpr int KT = C * DK / 2048, VT = C * DV / 2048;   // turns
#pragma unroll
  for (int u = 0; u < KT; ++u) {
    const int i = (tid + u * 512) * 4, r = i / DK, d = i % DK;
    const int left = r < n ? a.dim - d : 0;
    const int64_t at = (t0 + r) * a.G * a.dim + grp * a.dim + d;
    const float4 q = fetch(a.q + at, left, vec_k), k = fetch(a.k + at, left, vec_k);
    float4 g = fetch(a.logg + ((t0 + r) * a.H + h) * a.dim + d, left, vec_k);
    g = make_float4(g.x * kLog2e, g.y * kLog2e, g.z * kLog2e, g.w * kLog2e);
    store4(q_s + r * LD + d, q);
    store4(k_s + r * LD + d, k);
    store4(b_s + r * LD + d, g);
  }
  if (tid < C) be[tid] = tid < n ? a.beta[(t0 + tid) * a.H + h] : 0.0f;
  for (int i = tid; i < C * LT; i += 512) L_s[i] = X_s[i] = 0.0f;
  __syncthreads();
  {   // running sums: SEG row segments per channel
    constexpr int SEG = 512 / DK, ROWS = C / SEG;
    const int d = tid % DK, sg = tid / DK;
    float s = 0.0f;
    for (int r = 0; r < ROWS; ++r) s += b_s[(sg * ROWS + r) * LD + d];
    kx[sg * DK + d] = s;
    __syncthreads();
    float run = 0.0f;
    for (int e = 0; e < sg; ++e) run += kx[e * DK + d];
    for (int r = 0; r < ROWS; ++r) {
      float* p = b_s + (sg * ROWS + r) * LD + d;
      run += *p;
      *p = run;
    }
    __syncthreads();
  }
  float* B = a.scores + tile * (C * C);
  // pairs in different 16-row blocks
  for (int I = 1; I < 4; ++I) {
    const float* ref = b_s + (16 * I - 1) * LD;
    for (int i = tid * 4; i < 16 * (I + 1) * DK; i += 2048) {   // rows before the block, then its own
      const int r = i / DK, d = i % DK;
      const float4 z = ld4(ref + d), b = ld4(b_s + r * LD + d), k = ld4(k_s + r * LD + d);
      if (r < 16 * I) {
        store4(kx + r * LD + d, make_float4(k.x * ex2(z.x - b.x), k.y * ex2(z.y - b.y), k.z * ex2(z.z - b.z), k.w * ex2(z.w - b.w)));
      } else {
        const float4 q = ld4(q_s + r * LD + d);
        const float4 e = make_float4(ex2(b.x - z.x), ex2(b.y - z.y), ex2(b.z - z.z), ex2(b.w - z.w));
        store4(kr + (r - 16 * I) * LD + d, make_float4(k.x * e.x, k.y * e.y, k.z * e.z, k.w * e.w));
        store4(qr + (r - 16 * I) * LD + d, make_float4(q.x * e.x, q.y * e.y, q.z * e.z, q.w * e.w));
      }
    }
    __syncthreads();
    const int cols = 16 * I;
    for (int p = tid; p < 8 * cols; p += 512) {   // two rows per thread
      const int i0 = p / cols * 2, j = p % cols;
      float ka = 0.0f, kb = 0.0f, qa = 0.0f, qb = 0.0f;
#pragma unroll 4
      for (int d = 0; d < DK; d += 4) {
        const float4 x = ld4(kx + j * LD + d);
        ka = dot4(ld4(kr + i0 * LD + d), x, ka);
        kb = dot4(ld4(kr + (i0 + 1) * LD + d), x, kb);
        qa = dot4(ld4(qr + i0 * LD + d), x, qa);
        qb = dot4(ld4(qr + (i0 + 1) * LD + d), x, qb);
      }
      const int i = 16 * I + i0;
      L_s[i * LT + j] = be[i] * ka;
      L_s[(i + 1) * LT + j] = be[i + 1] * kb;
      B[i * C + j] = qa;
      B[(i + 1) * C + j] = qb;
    }
    __syncthreads();
  }
  {   // pairs inside a block: four columns per item, two threads share the channels
    // A warp takes four neighbouring rows i and only the column steps u that reach below their diagonal;
    // the row groups are dealt so that every scheduler gets long and short ones.
    const int half = tid & 1, jq = (tid >> 1) & 3, w = tid >> 5;
    const int blk = w >> 2 << 4, ig = ((w >> 2) + w) & 3, i = blk + 4 * ig + ((tid >> 3) & 3);
    float ak[4] = {0, 0, 0, 0}, aq[4] = {0, 0, 0, 0};
    {
#pragma unroll 2
      for (int d = half * 4; d < DK; d += 8) {
        const float4 bi = ld4(b_s + i * LD + d), ki = ld4(k_s + i * LD + d), qi = ld4(q_s + i * LD + d);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (u > ig) break;
          const int j = blk + jq + 4 * u;
          const float4 bj = ld4(b_s + j * LD + d), kj = ld4(k_s + j * LD + d);
          const float e0 = kj.x * ex2(bi.x - bj.x), e1 = kj.y * ex2(bi.y - bj.y), e2 = kj.z * ex2(bi.z - bj.z),
                      e3 = kj.w * ex2(bi.w - bj.w);
          ak[u] = fmaf(ki.x, e0, fmaf(ki.y, e1, fmaf(ki.z, e2, fmaf(ki.w, e3, ak[u]))));
          aq[u] = fmaf(qi.x, e0, fmaf(qi.y, e1, fmaf(qi.z, e2, fmaf(qi.w, e3, aq[u]))));
        }
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      ak[u] += __shfl_xor_sync(0xffffffffu, ak[u], 1);
      aq[u] += __shfl_xor_sync(0xffffffffu, aq[u], 1);
      const int j = blk + jq + 4 * u;
      if (half == 0) {
        if (j < i) L_s[i * LT + j] = be[i] * ak[u];
        B[i * C + j] = j <= i ? aq[u] : 0.0f;   // above the diagonal e^(b_i - b_j) may have overflowed: not used
      }
    }
    for (int p = tid; p < C * C; p += 512)
      if ((p % C) / 16 > (p / C) / 16) B[p] = 0.0f;
  }
  __syncthreads();
  // X = (I + L)^-1: the 16 x 16 diagonal blocks by forward substitution, one column per thread
  if (tid < C) {
    const int blk = tid & ~15, col = tid & 15;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float s = r == col ? 1.0f : 0.0f;
#pragma unroll
      for (int e = 0; e < r; ++e) s = fmaf(-L_s[(blk + r) * LT + blk + e], x[e], s);
      x[r] = s;   // zero above the diagonal: every term is
    }
#pragma unroll
    for (int r = 0; r < 16; ++r) X_s[(blk + r) * LT + blk + col] = x[r];
  }
  __syncthreads();
  for (int d = 1; d < 4; ++d) {   // block diagonals below: X_ij = -X_ii sum_k L_ik X_kj
    const int nb = 4 - d;
    for (int p = tid; p < nb * 256; p += 512) {
      const int j = p >> 8, i = j + d, r = (p >> 4) & 15, col = p & 15;
      float s = 0.0f;
      for (int k = 16 * j; k < 16 * i; ++k) s = fmaf(L_s[(16 * i + r) * LT + k], X_s[k * LT + 16 * j + col], s);
      tmp[(j * 16 + r) * 17 + col] = s;
    }
    __syncthreads();
    for (int p = tid; p < nb * 256; p += 512) {
      const int j = p >> 8, i = j + d, r = (p >> 4) & 15, col = p & 15;
      float s = 0.0f;
#pragma unroll
      for (int e = 0; e < 16; ++e) s = fmaf(X_s[(16 * i + r) * LT + 16 * i + e], tmp[(j * 16 + e) * 17 + col], s);
      X_s[(16 * i + r) * LT + 16 * j + col] = -s;
    }
    __syncthreads();
  }
  for (int p = tid; p < C * C; p += 512) X_s[(p / C) * LT + p % C] *= be[p % C];
  // what the state and output kernels multiply with; the values replace q
  float4 val[VT];
#pragma unroll
  for (int u = 0; u < VT; ++u) {
    const int i = (tid + u * 512) * 4, r = i / DV, d = i % DV;
    val[u] = fetch(a.v + (t0 + r) * a.H * a.vdim + h * a.vdim + d, r < n ? a.vdim - d : 0, vec_v);
  }
#pragma unroll
  for (int u = 0; u < KT; ++u) {
    const int i = (tid + u * 512) * 4, r = i / DK, d = i % DK;
    const float4 b = ld4(b_s + r * LD + d), k = ld4(k_s + r * LD + d), q = ld4(q_s + r * LD + d), z = ld4(b_s + (C - 1) * LD + d);
    const float4 e = make_float4(ex2(b.x), ex2(b.y), ex2(b.z), ex2(b.w));
    put4<SPLIT>(a.kh + tile * (C * DK), C * DK, i,
                make_float4(k.x * ex2(z.x - b.x), k.y * ex2(z.y - b.y), k.z * ex2(z.z - b.z), k.w * ex2(z.w - b.w)));
    put4<SPLIT>(a.qt + tile * (C * DK), C * DK, i, make_float4(q.x * e.x, q.y * e.y, q.z * e.z, q.w * e.w));
    store4(k_s + r * LD + d, make_float4(k.x * e.x, k.y * e.y, k.z * e.z, k.w * e.w));
    if (r == C - 1) store4(a.decay + tile * DK + d, e);
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < VT; ++u) {
    const int i = (tid + u * 512) * 4, r = i / DV, d = i % DV;
    store4(q_s + r * LV + d, val[u]);
  }
  __syncthreads();
  for (int it = tid; it < 16 * (DK / 4); it += 512) {
    const int r0 = it / (DK / 4) * 4, c0 = it % (DK / 4) * 4;
    float acc[4][4] = {};
    tile_product(X_s, LT, k_s, LD, r0, c0, r0 + 4, acc);
#pragma unroll
    for (int r = 0; r < 4; ++r)
      put4<SPLIT>(a.w + tile * (C * DK), C * DK, (r0 + r) * DK + c0, make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]));
  }
  for (int it = tid; it < 16 * (DV / 4); it += 512) {
    const int r0 = it / (DV / 4) * 4, c0 = it % (DV / 4) * 4;
    float acc[4][4] = {};
    tile_product(X_s, LT, q_s, LV, r0, c0, r0 + 4, acc);
#pragma unroll
    for (int r = 0; r < 4; ++r)
      *reinterpret_cast<float4*>(a.u + tile * (C * DV) + (r0 + r) * DV + c0) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
  }
}

constexpr int NB = 16;        // value columns of a state CTA
constexpr int LN = NB + 4;

template <int DK>
struct StateCfg {
  static constexpr int LD = DK + 4;
  static constexpr int kStage = 2 * C * LD + C * LN + DK;
  static constexpr int kFloats = 2 * kStage + DK * LN + C * LN;
};

// grid (DV / 16, heads), 512 threads: U = T V - W S and the state, chunk after chunk.
constexpr int kStateThreads = 512;
template <int DK, int DV>
__global__ void __launch_bounds__(kStateThreads, 1) delta_state_kernel(const DeltaChunkArgs a, int chunks) {
  using Cfg = StateCfg<DK>;
  constexpr int LD = Cfg::LD;
  extern __shared__ __align__(16) float sm[];
  float* S_s = sm + 2 * Cfg::kStage;   // [DK][LN]
  float* U_s = S_s + DK * LN;          // [C][LN]
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.y, c0 = blockIdx.x * NB, tid = threadIdx.x;
  auto load = [&](int c) {
    float* st = sm + (c & 1) * Cfg::kStage;
    const int64_t tile = static_cast<int64_t>(c) * a.H + h;
    const float* w = a.w + tile * (C * DK);
    const float* kh = a.kh + tile * (C * DK);
    for (int i = tid; i < C * (DK / 4); i += kStateThreads) {
      const int r = i / (DK / 4), p = i % (DK / 4) * 4;
      cp_async16(st + r * LD + p, w + r * DK + p);
      cp_async16(st + (C + r) * LD + p, kh + r * DK + p);
    }
    float* us = st + 2 * C * LD;
    if (tid < C * 4) {
      const int r = tid >> 2, p = (tid & 3) * 4;
      cp_async16(us + r * LN + p, a.u + tile * (C * DV) + r * DV + c0 + p);
    }
    if (tid < DK / 4) cp_async16(us + C * LN + tid * 4, a.decay + tile * DK + tid * 4);
    cp_async_commit();
  };
  // a thread owns state rows k0, k0 + 1, columns s0, s0 + 1
  const int k0 = tid / 8 * 2, s0 = (tid & 7) * 2;
  const bool owner = k0 < DK;
  float S[2][2] = {};
  if (owner) {
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int r = k0 + e, col = c0 + s0 + f;
        if (a.resume && r < a.dim && col < a.vdim) S[e][f] = a.state[(static_cast<int64_t>(h) * a.dim + r) * a.vdim + col];
        S_s[r * LN + s0 + f] = S[e][f];
      }
  }
  load(0);
  // for U: row ur, columns uc .. uc + 3, and half of the key channels (neighbouring lanes add up)
  const int ur = tid >> 3, uc = ((tid >> 1) & 3) * 4, kh2 = (tid & 1) * 4;
  for (int c = 0; c < chunks; ++c) {
    const int64_t tile = static_cast<int64_t>(c) * a.H + h;
    if (c + 1 < chunks) {
      load(c + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();   // this chunk's operands and the state have landed
    const float* W = sm + (c & 1) * Cfg::kStage;
    const float* Kh = W + C * LD;
    const float* Uv = Kh + C * LD;
    const float* dec = Uv + C * LN;
    if (owner)
#pragma unroll
      for (int e = 0; e < 2; ++e)
        *reinterpret_cast<float2*>(a.chunk_state + tile * (DK * DV) + (k0 + e) * DV + c0 + s0) = make_float2(S[e][0], S[e][1]);
    float u[4] = {}, u2[4] = {};
#pragma unroll 8
    for (int k = kh2; k < DK; k += 8) {
      const float4 w = ld4(W + ur * LD + k);
      axpy4(w.x, ld4(S_s + k * LN + uc), u);
      axpy4(w.y, ld4(S_s + (k + 1) * LN + uc), u2);
      axpy4(w.z, ld4(S_s + (k + 2) * LN + uc), u);
      axpy4(w.w, ld4(S_s + (k + 3) * LN + uc), u2);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      u[e] += u2[e];
      u[e] += __shfl_xor_sync(0xffffffffu, u[e], 1);
    }
    const float4 v = ld4(Uv + ur * LN + uc);
    const float4 res = make_float4(v.x - u[0], v.y - u[1], v.z - u[2], v.w - u[3]);
    if (kh2 == 0) store4(U_s + ur * LN + uc, res);
    else store4(a.u + tile * (C * DV) + ur * DV + c0 + uc, res);
    __syncthreads();
    if (owner) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float d = dec[k0 + e];
        S[e][0] *= d;
        S[e][1] *= d;
      }
#pragma unroll 8
      for (int j = 0; j < C; ++j) {
        const float2 k = *reinterpret_cast<const float2*>(Kh + j * LD + k0);
        const float2 x = *reinterpret_cast<const float2*>(U_s + j * LN + s0);
        S[0][0] = fmaf(k.x, x.x, S[0][0]);
        S[0][1] = fmaf(k.x, x.y, S[0][1]);
        S[1][0] = fmaf(k.y, x.x, S[1][0]);
        S[1][1] = fmaf(k.y, x.y, S[1][1]);
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) *reinterpret_cast<float2*>(S_s + (k0 + e) * LN + s0) = make_float2(S[e][0], S[e][1]);
    }
    __syncthreads();   // nobody reads this stage or the old state any more
  }
  if (owner) {
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int r = k0 + e, col = c0 + s0 + f;
        if (r < a.dim && col < a.vdim) a.state[(static_cast<int64_t>(h) * a.dim + r) * a.vdim + col] = S[e][f];
      }
  }
}

template <int DK>
struct OutCfg {
  static constexpr int LD = DK + 4, LB = 64 + 4;
  static constexpr int kFloats = C * LD + DK * LB + C * LT + C * LB;
};

// grid (chunks, heads, DV / 64), 256 threads.
template <int DK, int DV>
__global__ void __launch_bounds__(256) delta_out_kernel(const DeltaChunkArgs a) {
  using Cfg = OutCfg<DK>;
  constexpr int LD = Cfg::LD, LB = Cfg::LB;
  extern __shared__ __align__(16) float sm[];
  float* Q = sm;                // [C][LD]
  float* S = Q + C * LD;        // [DK][LB]
  float* B = S + DK * LB;       // [C][LT]
  float* U = B + C * LT;        // [C][LB]
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, n0 = blockIdx.z * 64, tid = threadIdx.x;
  const int64_t t0 = static_cast<int64_t>(c) * C, tile = static_cast<int64_t>(c) * a.H + h;
  auto copy = [&](float* dst, int ld, const float* src, int lds, int rows, int cols) {
    const int per = cols / 4;
    for (int i = tid; i < rows * per; i += 256) cp_async16(dst + i / per * ld + i % per * 4, src + static_cast<int64_t>(i / per) * lds + i % per * 4);
  };
  copy(Q, LD, a.qt + tile * (C * DK), DK, C, DK);
  copy(S, LB, a.chunk_state + tile * (DK * DV) + n0, DV, DK, 64);
  copy(B, LT, a.scores + tile * (C * C), C, C, C);
  copy(U, LB, a.u + tile * (C * DV) + n0, DV, C, 64);
  cp_async_commit();
  cp_async_wait_all();
  __syncthreads();
  const int r0 = tid / 16 * 4, c0 = (tid & 15) * 4;
  float acc[4][4] = {};
  tile_product(Q, LD, S, LB, r0, c0, DK, acc);
  tile_product(B, LT, U, LB, r0, c0, r0 + 4, acc);
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (r0 + r < n && n0 + c0 + e < a.vdim) a.out[(t0 + r0 + r) * a.H * a.vdim + h * a.vdim + n0 + c0 + e] = acc[r][e];
}

// ---- split form ----
constexpr int LNB = NB + 8;   // bfloat16 pitch of the 16-column tiles

template <int DK>
struct SplitStateCfg {
  static constexpr int LK = DK + 8;
  static constexpr int kStage = 4 * C * LK * 2 + C * LN * 4 + DK * 4;   // W high / low, K high / low, T V, decay (bytes)
  static constexpr int kBytes = 2 * kStage + 2 * DK * LNB * 2 + 2 * C * LNB * 2;
};

// grid (DV / 16, heads), 256 threads. A warp owns one (16-row, 8-column) tile of U and 16 rows of the
// state, which stays in its accumulators.
template <int DK, int DV>
__global__ void __launch_bounds__(256, 1) delta_state_split_kernel(const DeltaChunkArgs a, int chunks) {
  using Cfg = SplitStateCfg<DK>;
  constexpr int LK = Cfg::LK;
  extern __shared__ __align__(16) unsigned char raw[];
  __nv_bfloat16* Sh = reinterpret_cast<__nv_bfloat16*>(raw + 2 * Cfg::kStage);   // [DK][LNB]
  __nv_bfloat16* Sl = Sh + DK * LNB;
  __nv_bfloat16* Uh = Sl + DK * LNB;   // [C][LNB]
  __nv_bfloat16* Ul = Uh + C * LNB;
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.y, c0 = blockIdx.x * NB, tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  auto load = [&](int c) {
    unsigned char* st = raw + (c & 1) * Cfg::kStage;
    __nv_bfloat16* ops = reinterpret_cast<__nv_bfloat16*>(st);   // four planes [C][LK]
    const int64_t tile = static_cast<int64_t>(c) * a.H + h;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.w + tile * (C * DK));
    const __nv_bfloat16* kh = reinterpret_cast<const __nv_bfloat16*>(a.kh + tile * (C * DK));
#pragma unroll
    for (int i = tid; i < 2 * C * (DK / 8); i += 256) {   // both planes are contiguous rows
      const int r = i / (DK / 8), p = i % (DK / 8) * 8;
      cp_async16(ops + r * LK + p, w + r * DK + p);
      cp_async16(ops + (2 * C + r) * LK + p, kh + r * DK + p);
    }
    float* us = reinterpret_cast<float*>(st + 4 * C * LK * 2);
    const int r = tid >> 2, p = (tid & 3) * 4;
    cp_async16(us + r * LN + p, a.u + tile * (C * DV) + r * DV + c0 + p);
    if (tid < DK / 4) cp_async16(us + C * LN + tid * 4, a.decay + tile * DK + tid * 4);
    cp_async_commit();
  };
  // accumulator element e of column tile t: row wid * 16 + lane / 4 + (e / 2) * 8, column t * 8 + (lane % 4) * 2 + e % 2
  const int sr = wid * 16 + (lane >> 2), sc = (lane & 3) * 2;
  const bool owner = wid * 16 < DK;
  float S[2][4];
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = sr + (e >> 1) * 8, col = c0 + t * 8 + sc + (e & 1);
      S[t][e] = (a.resume && owner && r < a.dim && col < a.vdim) ? a.state[(static_cast<int64_t>(h) * a.dim + r) * a.vdim + col] : 0.0f;
    }
  load(0);
  for (int c = 0; c < chunks; ++c) {
    const int64_t tile = static_cast<int64_t>(c) * a.H + h;
    if (owner) {   // the state in front of the chunk: for this chunk's products, and for the output kernel
      __nv_bfloat16* g = reinterpret_cast<__nv_bfloat16*>(a.chunk_state + tile * (DK * DV));
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int f = 0; f < 2; ++f) {
          const int r = sr + f * 8, col = t * 8 + sc;
          uint32_t hi, lo;
          split_bf16x2(S[t][2 * f], S[t][2 * f + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(Sh + r * LNB + col) = hi;
          *reinterpret_cast<uint32_t*>(Sl + r * LNB + col) = lo;
          *reinterpret_cast<uint32_t*>(g + r * (2 * DV) + c0 + col) = hi;
          *reinterpret_cast<uint32_t*>(g + r * (2 * DV) + DV + c0 + col) = lo;
        }
    }
    if (c + 1 < chunks) {
      load(c + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();   // operands and state have landed
    const unsigned char* st = raw + (c & 1) * Cfg::kStage;
    const __nv_bfloat16* Wh = reinterpret_cast<const __nv_bfloat16*>(st);
    const __nv_bfloat16* Wl = Wh + C * LK;
    const __nv_bfloat16* Kh = Wl + C * LK;
    const __nv_bfloat16* Kl = Kh + C * LK;
    const float* Uv = reinterpret_cast<const float*>(st + 4 * C * LK * 2);
    const float* dec = Uv + C * LN;
    {
      const int m0 = (wid & 3) * 16, nt = wid >> 2;
      float p[3][4] = {};
#pragma unroll
      for (int k0 = 0; k0 < DK; k0 += 16) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldsm_a(ah, Wh, LK, m0, k0, lane);
        ldsm_a(al, Wl, LK, m0, k0, lane);
        ldsm_b_trans(bh, Sh, LNB, k0, 0, lane);
        ldsm_b_trans(bl, Sl, LNB, k0, 0, lane);
        const uint32_t h0 = nt ? bh[2] : bh[0], h1 = nt ? bh[3] : bh[1], l0 = nt ? bl[2] : bl[0], l1 = nt ? bl[3] : bl[1];
        mma_bf16(p[0], ah, h0, h1);
        mma_bf16(p[1], ah, l0, l1);
        mma_bf16(p[2], al, h0, h1);
      }
      __nv_bfloat16* gu = reinterpret_cast<__nv_bfloat16*>(a.us + tile * (C * DV));
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int r = m0 + (lane >> 2) + f * 8, col = nt * 8 + sc;
        const float2 v = *reinterpret_cast<const float2*>(Uv + r * LN + col);
        const float x = v.x - (p[0][2 * f] + (p[1][2 * f] + p[2][2 * f])), y = v.y - (p[0][2 * f + 1] + (p[1][2 * f + 1] + p[2][2 * f + 1]));
        uint32_t hi, lo;
        split_bf16x2(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(Uh + r * LNB + col) = hi;
        *reinterpret_cast<uint32_t*>(Ul + r * LNB + col) = lo;
        *reinterpret_cast<uint32_t*>(gu + r * DV + c0 + col) = hi;
        *reinterpret_cast<uint32_t*>(gu + C * DV + r * DV + c0 + col) = lo;
      }
    }
    __syncthreads();
    if (owner) {
      float q[2][2][4] = {};   // the cross terms, summed apart from the state
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[t][e] *= dec[sr + (e >> 1) * 8];
#pragma unroll
      for (int k0 = 0; k0 < C; k0 += 16) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldsm_a_trans(ah, Kh, LK, wid * 16, k0, lane);
        ldsm_a_trans(al, Kl, LK, wid * 16, k0, lane);
        ldsm_b_trans(bh, Uh, LNB, k0, 0, lane);
        ldsm_b_trans(bl, Ul, LNB, k0, 0, lane);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma_bf16(S[t], ah, bh[2 * t], bh[2 * t + 1]);
          mma_bf16(q[0][t], ah, bl[2 * t], bl[2 * t + 1]);
          mma_bf16(q[1][t], al, bh[2 * t], bh[2 * t + 1]);
        }
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[t][e] += q[0][t][e] + q[1][t][e];
    }
    __syncthreads();   // nobody reads this stage, the old state or U any more
  }
  if (owner) {
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = sr + (e >> 1) * 8, col = c0 + t * 8 + sc + (e & 1);
        if (r < a.dim && col < a.vdim) a.state[(static_cast<int64_t>(h) * a.dim + r) * a.vdim + col] = S[t][e];
      }
  }
}

template <int DK>
struct SplitOutCfg {
  static constexpr int LK = DK + 8, LB = 64 + 8;
  static constexpr int kBytes = (2 * C * LK + 2 * DK * LB + 2 * C * LB) * 2;
};

// grid (chunks, heads, DV / 64), 128 threads: a warp owns 16 rows and 64 columns.
template <int DK, int DV>
__global__ void __launch_bounds__(128) delta_out_split_kernel(const DeltaChunkArgs a) {
  using Cfg = SplitOutCfg<DK>;
  constexpr int LK = Cfg::LK, LB = Cfg::LB;
  extern __shared__ __align__(16) unsigned char raw[];
  __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(raw);   // [2][C][LK]
  __nv_bfloat16* S = Q + 2 * C * LK;                          // [2][DK][LB]
  __nv_bfloat16* U = S + 2 * DK * LB;                         // [2][C][LB]
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, n0 = blockIdx.z * 64, tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const int64_t t0 = static_cast<int64_t>(c) * C, tile = static_cast<int64_t>(c) * a.H + h;
  auto copy = [&](__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, int lds, int rows, int cols) {
    const int per = cols / 8;
    for (int i = tid; i < rows * per; i += 128) cp_async16(dst + i / per * ld + i % per * 8, src + static_cast<int64_t>(i / per) * lds + i % per * 8);
  };
  const __nv_bfloat16* gs = reinterpret_cast<const __nv_bfloat16*>(a.chunk_state + tile * (DK * DV));
  copy(Q, LK, reinterpret_cast<const __nv_bfloat16*>(a.qt + tile * (C * DK)), DK, 2 * C, DK);
  copy(S, LB, gs + n0, 2 * DV, DK, 64);
  copy(S + DK * LB, LB, gs + DV + n0, 2 * DV, DK, 64);
  copy(U, LB, reinterpret_cast<const __nv_bfloat16*>(a.us + tile * (C * DV)) + n0, DV, 2 * C, 64);
  cp_async_commit();
  const int m0 = wid * 16, r0 = m0 + (lane >> 2);
  const float* B = a.scores + tile * (C * C);
  float2 sc[C / 16][4];   // scores of the warp's rows, in the order of an A fragment
#pragma unroll
  for (int kk = 0; kk < C / 16; ++kk)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      sc[kk][e] = kk * 16 < m0 + 16 ? *reinterpret_cast<const float2*>(B + (r0 + (e & 1) * 8) * C + kk * 16 + (e >> 1) * 8 + (lane & 3) * 2)
                                    : make_float2(0.0f, 0.0f);
  cp_async_wait_all();
  __syncthreads();
  float o[8][4] = {};
#pragma unroll 2
  for (int k0 = 0; k0 < DK; k0 += 16) {
    uint32_t ah[4], al[4], bh[4], bl[4];
    ldsm_a(ah, Q, LK, m0, k0, lane);
    ldsm_a(al, Q + C * LK, LK, m0, k0, lane);
#pragma unroll
    for (int t = 0; t < 8; t += 2) {
      ldsm_b_trans(bh, S, LB, k0, t * 8, lane);
      ldsm_b_trans(bl, S + DK * LB, LB, k0, t * 8, lane);
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        mma_bf16(o[t + f], ah, bh[2 * f], bh[2 * f + 1]);
        mma_bf16(o[t + f], ah, bl[2 * f], bl[2 * f + 1]);
        mma_bf16(o[t + f], al, bh[2 * f], bh[2 * f + 1]);
      }
    }
  }
#pragma unroll
  for (int kk = 0; kk < C / 16; ++kk) {
    if (kk * 16 >= m0 + 16) break;
    uint32_t ah[4], al[4], bh[4], bl[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) split_bf16x2(sc[kk][e].x, sc[kk][e].y, ah[e], al[e]);
#pragma unroll
    for (int t = 0; t < 8; t += 2) {
      ldsm_b_trans(bh, U, LB, kk * 16, t * 8, lane);
      ldsm_b_trans(bl, U + C * LB, LB, kk * 16, t * 8, lane);
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        mma_bf16(o[t + f], ah, bh[2 * f], bh[2 * f + 1]);
        mma_bf16(o[t + f], ah, bl[2 * f], bl[2 * f + 1]);
        mma_bf16(o[t + f], al, bh[2 * f], bh[2 * f + 1]);
      }
    }
  }
  const int n = static_cast<int>(a.rows - t0 < C ? a.rows - t0 : C);
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
int launch_split(const DeltaChunkArgs& a, cudaStream_t s) {
  const int chunks = static_cast<int>((a.rows + C - 1) / C);
  constexpr size_t m1 = LocalCfg<DK, DV>::kFloats * 4, m2 = SplitStateCfg<DK>::kBytes, m3 = SplitOutCfg<DK>::kBytes;
  static_assert(m1 <= 227 * 1024 && m2 <= 227 * 1024, "shared memory");
  cudaError_t e = cudaFuncSetAttribute(delta_local_kernel<DK, DV, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m1));
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(delta_state_split_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m2));
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(delta_out_split_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m3));
  if (e == cudaSuccess) e = launch_pdl(delta_local_kernel<DK, DV, true>, dim3(chunks, a.H), dim3(512), m1, s, a);
  if (e == cudaSuccess) e = launch_pdl(delta_state_split_kernel<DK, DV>, dim3(DV / NB, a.H), dim3(256), m2, s, a, chunks);
  if (e == cudaSuccess) e = launch_pdl(delta_out_split_kernel<DK, DV>, dim3(chunks, a.H, DV / 64), dim3(128), m3, s, a);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "delta chunks: %s", cudaGetErrorString(e));
  check_launch("delta chunks");
  check_launch("delta chunks");
  return check_launch("delta chunks");
}

template <int DK, int DV>
int launch(const DeltaChunkArgs& a, cudaStream_t s) {
  const int chunks = static_cast<int>((a.rows + C - 1) / C);
  constexpr size_t m1 = LocalCfg<DK, DV>::kFloats * 4, m2 = StateCfg<DK>::kFloats * 4, m3 = OutCfg<DK>::kFloats * 4;
  static_assert(m1 <= 227 * 1024 && m2 <= 227 * 1024, "shared memory");
  cudaError_t e = cudaFuncSetAttribute(delta_local_kernel<DK, DV, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m1));
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(delta_state_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m2));
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(delta_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(m3));
  if (e == cudaSuccess) e = launch_pdl(delta_local_kernel<DK, DV, false>, dim3(chunks, a.H), dim3(512), m1, s, a);
  if (e == cudaSuccess) e = launch_pdl(delta_state_kernel<DK, DV>, dim3(DV / NB, a.H), dim3(kStateThreads), m2, s, a, chunks);
  if (e == cudaSuccess) e = launch_pdl(delta_out_kernel<DK, DV>, dim3(chunks, a.H, DV / 64), dim3(256), m3, s, a);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "delta chunks: %s", cudaGetErrorString(e));
  check_launch("delta chunks");
  check_launch("delta chunks");
  return check_launch("delta chunks");
}

}  // namespace

bool delta_chunked_ok(int dim, int vdim) { return dim <= 128 && vdim <= 128; }

int delta_chunked(const DeltaChunkArgs& a, cudaStream_t s) {
  CTDK_REQUIRE(delta_chunked_ok(a.dim, a.vdim) && a.H <= 65535, "delta chunks: head sizes above 128");
  const int dk = lightning_tile(a.dim), dv = lightning_tile(a.vdim);
  if (a.split) {
    if (dk == 64) return dv == 64 ? launch_split<64, 64>(a, s) : launch_split<64, 128>(a, s);
    return dv == 64 ? launch_split<128, 64>(a, s) : launch_split<128, 128>(a, s);
  }
  if (dk == 64) return dv == 64 ? launch<64, 64>(a, s) : launch<64, 128>(a, s);
  return dv == 64 ? launch<128, 64>(a, s) : launch<128, 128>(a, s);
}

}  // namespace hybrid
}  // namespace ctdk
