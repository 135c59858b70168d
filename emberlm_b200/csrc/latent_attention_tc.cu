// Causal latent attention of a prompt's portion on the tcgen05 tensor cores, bfloat16 operands, fp32 scores
// and sums. A query attends with two parts: the unrotated one against its head's keys (read out of the
// latents into one buffer), the rotated one against the key part that all heads share (read in place from the
// latent cache); both products go into the same accumulator.
//
// Persistent CTAs, one per SM, walk a list of (128-query tile, head) items, longest first. 6 warps:
//   warp 0    TMA producer: Q once per item, then steps of 128 keys (unrotated chunks, rotated chunk) and
//             values through two-stage rings; 3-D maps with a head's width as the inner extent, so that the
//             columns up to the 64-wide chunk come in as zeros.
//   warp 1    MMA issuer: S(j) = Q K(j)^T into one of two 128-column buffers in tensor memory; O += P(j) V(j)
//             with P from tensor memory (two bfloat16 per column, over S) and V as an MN-major operand.
//             S(j+2) is queued right behind P V(j).
//   warps 2-5 softmax: one query row per thread, exponentials in the log2 domain, O rescaled lazily (only
//             when a row's maximum grew by more than 2^8), head gate and normalisation at the end.
// Every mbarrier wait is bounded.
#include <cfloat>
#include <climits>

#include "hybrid_kernels.h"
#include "parallel_kernels.h"

namespace ctdk {
namespace hybrid {
namespace {

constexpr int TQ = 128, TKEY = 128;
constexpr int kChunk = 128 * 128;   // bytes of a {64 columns x 128 rows} box
constexpr float kLog2e = 1.4426950408889634f, kSlack = 8.0f;

template <int NCN, int NV>
struct Cfg {
  static constexpr int kQBytes = (NCN + 1) * kChunk, kKBytes = (NCN + 1) * kChunk, kVBytes = NV * kChunk;
  static constexpr int kSmem = kQBytes + 2 * kKBytes + 2 * kVBytes + 1024 + 256;
};

struct TcArgs {
  const float* gate;      // [rows, ld_gate] one column per head
  __nv_bfloat16* out;     // [rows, ld_out]
  int64_t ld_gate, ld_out;
  int rows, first, H, dim, rot_dim, vdim, n_items;
  float scale_log2;
  int* status;
};
struct Item {
  int h, q0, n_steps;
};
__device__ __forceinline__ Item item_at(const TcArgs& a, int it) {
  const int tiles = (a.rows + TQ - 1) / TQ;
  Item w;
  w.h = it % a.H;
  w.q0 = (tiles - 1 - it / a.H) * TQ;
  const int last = a.first + min(w.q0 + TQ, a.rows);   // keys that the tile's last row sees
  w.n_steps = (last + TKEY - 1) / TKEY;
  return w;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ uint32_t idesc_bf16(bool b_mn, int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(b_mn) << 16) | (static_cast<uint32_t>(n >> 3) << 17) |
         (static_cast<uint32_t>(TQ >> 4) << 24);
}

template <int NCN, int NV>
__global__ void __launch_bounds__(192, 1)
    latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_qr,
                          const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_kr,
                          const __grid_constant__ CUtensorMap tm_v, const TcArgs a) {
  using C = Cfg<NCN, NV>;
  extern __shared__ unsigned char smem_raw[];
  pdl_launch();
  const uint32_t raw = smem_u32(smem_raw);
  unsigned char* smem = smem_raw + ((1024u - (raw & 1023u)) & 1023u);
  unsigned char* q_s = smem;
  unsigned char* k_s = q_s + C::kQBytes;       // [2] stages: unrotated chunks, then the rotated one
  unsigned char* v_s = k_s + 2 * C::kKBytes;   // [2] stages
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + 2 * C::kVBytes);
  uint64_t* q_full = bars;          // one phase per item
  uint64_t* q_empty = bars + 1;     // every score product of the item has read Q
  uint64_t* k_full = bars + 2;      // [2] stage / phase by the running step count
  uint64_t* k_empty = bars + 4;
  uint64_t* v_full = bars + 6;
  uint64_t* v_empty = bars + 8;
  uint64_t* s_full = bars + 10;     // S(g) is in tensor memory
  uint64_t* p_ready = bars + 12;    // P(g) has replaced S(g) (128 arrivals)
  uint64_t* pv_full = bars + 14;    // O += P(g) V(g) has finished (one phase per step)
  uint64_t* o_full = bars + 15;     // the item's last one has (one phase per item)
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 16; ++i) mbar_init(&bars[i], i == 12 || i == 13 ? 128 : 1);
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_qr);
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_kr);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
    tc_fence_before();
  }
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_wait();
  const uint32_t tm_o = tmem_base + 2u * TKEY;
  // g = running count of key steps over all items of this CTA: stage g & 1, phase (g >> 1) & 1
  if (warp == 0) {
    if (lane == 0) {
      uint32_t g0 = 0, n_it = 0;
      bool ok = true;
      for (int it = blockIdx.x; it < a.n_items && ok; it += gridDim.x) {
        const Item w = item_at(a, it);
        if (!mbar_wait_bounded(q_empty, (n_it & 1u) ^ 1u, a.status, 110)) break;
        ++n_it;
        mbar_expect_tx(q_full, C::kQBytes);
#pragma unroll
        for (int c = 0; c < NCN; ++c) tma_load_3d(q_s + c * kChunk, &tm_q, q_full, 64 * c, w.h, w.q0);
        tma_load_3d(q_s + NCN * kChunk, &tm_qr, q_full, 0, w.h, w.q0);
        auto load_k = [&](int j) {
          const uint32_t g = g0 + static_cast<uint32_t>(j), s = g & 1u;
          if (!mbar_wait_bounded(&k_empty[s], ((g >> 1) & 1u) ^ 1u, a.status, 111)) return false;
          mbar_expect_tx(&k_full[s], C::kKBytes);
          unsigned char* dst = k_s + s * C::kKBytes;
#pragma unroll
          for (int c = 0; c < NCN; ++c) tma_load_3d(dst + c * kChunk, &tm_k, &k_full[s], 64 * c, w.h, j * TKEY);
          tma_load_2d(dst + NCN * kChunk, &tm_kr, &k_full[s], 0, j * TKEY);
          return true;
        };
        auto load_v = [&](int j) {
          const uint32_t g = g0 + static_cast<uint32_t>(j), s = g & 1u;
          if (!mbar_wait_bounded(&v_empty[s], ((g >> 1) & 1u) ^ 1u, a.status, 112)) return false;
          mbar_expect_tx(&v_full[s], C::kVBytes);
#pragma unroll
          for (int c = 0; c < NV; ++c) tma_load_3d(v_s + s * C::kVBytes + c * kChunk, &tm_v, &v_full[s], 64 * c, w.h, j * TKEY);
          return true;
        };
        ok = load_k(0);
        for (int j = 0; j < w.n_steps && ok; ++j) {   // K runs one step ahead of V
          if (j + 1 < w.n_steps) ok = load_k(j + 1);
          if (ok) ok = load_v(j);
        }
        g0 += static_cast<uint32_t>(w.n_steps);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // The whole warp runs this role converged; one elected lane issues each MMA / commit.
    const uint32_t idesc_s = idesc_bf16(false, TKEY), idesc_pv = idesc_bf16(true, (a.vdim + 15) / 16 * 16);
    const uint32_t k_base = smem_u32(k_s), v_base = smem_u32(v_s);
    const uint64_t qd = make_smem_desc(smem_u32(q_s), 16, 1024, kLayoutSw128);
    const int ns = (a.dim + 15) / 16, nr = (a.rot_dim + 15) / 16;
    uint32_t g0 = 0, n_it = 0;
    bool ok = true;
    for (int it = blockIdx.x; it < a.n_items && ok; it += gridDim.x) {
      const Item w = item_at(a, it);
      auto issue_s = [&](int j) {
        const uint32_t g = g0 + static_cast<uint32_t>(j), s = g & 1u;
        if (!mbar_wait_bounded_w(&k_full[s], (g >> 1) & 1u, a.status, 122)) return false;
        tc_fence_after();
        const uint64_t kd = make_smem_desc(k_base + s * C::kKBytes, 16, 1024, kLayoutSw128);
        const uint32_t ts = tmem_base + s * TKEY;
        // a slice of 16 columns is 32 bytes of the swizzled row; the address field counts 16-byte units
#pragma unroll
        for (int ks = 0; ks < NCN * 4; ++ks) {
          const uint64_t off = ((ks >> 2) * kChunk + (ks & 3) * 32) >> 4;
          if (ks < ns) umma_bf16_w(ts, qd + off, kd + off, idesc_s, ks != 0 ? 1u : 0u);
        }
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          const uint64_t off = (NCN * kChunk + ks * 32) >> 4;
          if (ks < nr) umma_bf16_w(ts, qd + off, kd + off, idesc_s, 1u);
        }
        umma_commit_w(&k_empty[s]);
        umma_commit_w(&s_full[s]);
        if (j == w.n_steps - 1) umma_commit_w(q_empty);   // the item's last use of Q
        return true;
      };
      if (!mbar_wait_bounded_w(q_full, n_it & 1u, a.status, 121)) break;
      ++n_it;
      tc_fence_after();
      ok = issue_s(0);
      if (ok && w.n_steps > 1) ok = issue_s(1);
      for (int j = 0; j < w.n_steps && ok; ++j) {
        const uint32_t g = g0 + static_cast<uint32_t>(j), s = g & 1u, ph = (g >> 1) & 1u;
        if (!mbar_wait_bounded_w(&p_ready[s], ph, a.status, 123)) {
          ok = false;
          break;
        }
        if (!mbar_wait_bounded_w(&v_full[s], ph, a.status, 124)) {
          ok = false;
          break;
        }
        tc_fence_after();
        // B: 16 key rows (two 8-row swizzle groups, SBO) of every 64-column chunk of V (LBO)
        const uint64_t vd = make_smem_desc(v_base + s * C::kVBytes, kChunk, 1024, kLayoutSw128);
        const uint32_t ts = tmem_base + s * TKEY, acc0 = j != 0 ? 1u : 0u;
#pragma unroll
        for (int ks = 0; ks < TKEY / 16; ++ks)
          umma_bf16_ta_w(tm_o, ts + static_cast<uint32_t>(ks * 8), vd + ((ks * 2048) >> 4), idesc_pv, ks != 0 ? 1u : acc0);
        umma_commit_w(&v_empty[s]);
        umma_commit_w(pv_full);
        if (j == w.n_steps - 1) umma_commit_w(o_full);
        if (j + 2 < w.n_steps) ok = issue_s(j + 2);
      }
      g0 += static_cast<uint32_t>(w.n_steps);
    }
    __syncwarp();
  } else {
    const int qd = warp & 3;   // tensor-memory lane quarter of this warp
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const float sc = a.scale_log2;
    const uint32_t to = tm_o + lane_off;
    uint32_t g0 = 0, n_done = 0;
    bool ok = true;
    for (int it = blockIdx.x; it < a.n_items && ok; it += gridDim.x) {
      const Item w = item_at(a, it);
      const int t = w.q0 + qd * 32 + lane, row = a.first + t;   // of the portion, of the sequence
      float m_ref = 0.0f, l_run = 0.0f;
      for (int j = 0; j < w.n_steps && ok; ++j) {
        const uint32_t g = g0 + static_cast<uint32_t>(j), s = g & 1u;
        if (!mbar_wait_bounded_w(&s_full[s], (g >> 1) & 1u, a.status, 131)) {
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t ts = tmem_base + s * TKEY + lane_off;
        float x[2][64];
        tmem_ld_32x64_nowait(ts, x[0]);
        tmem_ld_32x64_nowait(ts + 64, x[1]);
        tmem_wait_ld();
        if ((j + 1) * TKEY > a.first + w.q0 + 1) {   // a step that reaches past the first row's own position
          const int n_valid = row - j * TKEY + 1;    // may be <= 0
#pragma unroll
          for (int hf = 0; hf < 2; ++hf)
#pragma unroll
            for (int i = 0; i < 64; ++i) x[hf][i] = hf * 64 + i < n_valid ? x[hf][i] : -FLT_MAX;
        }
        float mx[4] = {x[0][0], x[0][1], x[1][0], x[1][1]};
#pragma unroll
        for (int i = 2; i < 64; i += 4)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            mx[2 * hf] = fmax3(mx[2 * hf], x[hf][i], x[hf][i + 1]);
            if (i + 3 < 64) mx[2 * hf + 1] = fmax3(mx[2 * hf + 1], x[hf][i + 2], x[hf][i + 3]);
          }
        const float mxs = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * sc;
        float c = 1.0f;
        bool grow = false;
        if (j == 0) {
          m_ref = mxs;   // step 0 holds position 0, which every row sees
        } else if (mxs > m_ref + kSlack) {
          c = ex2(m_ref - mxs);
          m_ref = mxs;
          grow = true;
        }
        if (__any_sync(0xffffffffu, grow)) {
          // P V(g-1) must have landed before the accumulator is touched; P V(g) cannot start before every
          // row has arrived at p_ready below
          if (!mbar_wait_bounded_w(pv_full, (g - 1u) & 1u, a.status, 132)) {
            ok = false;
            break;
          }
          tc_fence_after();
#pragma unroll 1
          for (int p = 0; p < NV * 2; ++p) {
            float o[32];
            tmem_ld_32x32(to + p * 32, o);
#pragma unroll
            for (int i = 0; i < 32; i += 2) fmul2(o[i], o[i + 1], o[i], o[i + 1], c, c);
            tmem_st_32x32(to + p * 32, *reinterpret_cast<uint32_t(*)[32]>(o));
            tmem_wait_st();
          }
          l_run *= c;
        }
        const float neg_m = -m_ref;
        float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          uint32_t pb[32];
#pragma unroll
          for (int i = 0; i < 64; i += 2) {
            float u, v;
            ffma2(u, v, x[hf][i], x[hf][i + 1], sc, sc, neg_m, neg_m);
            u = ex2(u);
            v = ex2(v);
            fadd2(s0, s1, s0, s1, u, v);
            pb[i >> 1] = pack_bf16(u, v);
          }
          tmem_st_32x32(ts + hf * 32, pb);
        }
        tmem_wait_st();
        tc_fence_before();
        mbar_arrive(&p_ready[s]);
        l_run += s0 + s1;
      }
      g0 += static_cast<uint32_t>(w.n_steps);
      // The item's last P V. The next item's first one cannot start before these threads have read O and
      // arrived at its p_ready.
      if (!ok || !mbar_wait_bounded_w(o_full, n_done & 1u, a.status, 133)) {
        ok = false;
        break;
      }
      ++n_done;
      tc_fence_after();
      const bool live = t < a.rows;
      const float f = live ? sigmoid_f(a.gate[t * a.ld_gate + w.h]) / l_run : 0.0f;
      __nv_bfloat16* dst = a.out + t * a.ld_out + static_cast<int64_t>(w.h) * a.vdim;
#pragma unroll 1
      for (int p = 0; p < NV * 2; ++p) {
        if (p * 32 >= a.vdim) break;   // uniform
        float o[32];
        tmem_ld_32x32(to + p * 32, o);   // warp-collective: rows past the end take part too
#pragma unroll
        for (int i = 0; i < 32; i += 8)
          if (live && p * 32 + i < a.vdim)
            *reinterpret_cast<uint4*>(dst + p * 32 + i) =
                make_uint4(pack_bf16(o[i] * f, o[i + 1] * f), pack_bf16(o[i + 2] * f, o[i + 3] * f), pack_bf16(o[i + 4] * f, o[i + 5] * f),
                           pack_bf16(o[i + 6] * f, o[i + 7] * f));
        __syncwarp();
      }
      tc_fence_before();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int NCN, int NV>
int launch(const CUtensorMap (&m)[5], const TcArgs& a, cudaStream_t s) {
  using C = Cfg<NCN, NV>;
  cudaError_t e = cudaFuncSetAttribute(latent_attn_tc_kernel<NCN, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmem);
  if (e == cudaSuccess)
    e = launch_pdl(latent_attn_tc_kernel<NCN, NV>, dim3(a.n_items < sm_count() ? a.n_items : sm_count()), dim3(192), C::kSmem, s, m[0], m[1], m[2],
                   m[3], m[4], a);
  if (e != cudaSuccess) return fail(CTDK_ELAUNCH, "latent attention (tcgen05): %s", cudaGetErrorString(e));
  return check_launch("latent attention (tcgen05)");
}

}  // namespace

bool latent_tcgen05_ok(int dim, int rot_dim, int vdim) {
  return dim <= 128 && dim % 8 == 0 && rot_dim <= 64 && vdim <= 128 && vdim % 8 == 0;
}

int latent_attention_tcgen05(const LatentArgs<__nv_bfloat16>& a, int64_t first, int64_t rows, cudaStream_t s) {
  CTDK_REQUIRE(latent_tcgen05_ok(a.dim, a.rot_dim, a.vdim) && rows > 0 && first + rows <= INT32_MAX / 2, "latent attention (tcgen05): bad shape");
  const uint64_t L = static_cast<uint64_t>(first + rows), n = static_cast<uint64_t>(rows), H = static_cast<uint64_t>(a.H);
  const uint64_t pitch = static_cast<uint64_t>(latent_q_pitch(a.dim, a.rot_dim)), dp = static_cast<uint64_t>((a.dim + 7) / 8 * 8), rp = pitch - dp;
  const uint64_t ldkv = static_cast<uint64_t>(a.ld_kv) * 2, dim = static_cast<uint64_t>(a.dim), vdim = static_cast<uint64_t>(a.vdim);
  const uint32_t box3[3] = {64u, 1u, 128u}, box2[2] = {64u, 128u};
  CUtensorMap m[5];
  const uint64_t dq[3] = {dp, H, n}, sq[2] = {pitch * 2, H * pitch * 2}, dqr[3] = {rp, H, n};
  const uint64_t dk[3] = {dim, H, L}, sk[2] = {dim * 2, ldkv}, dkr[2] = {rp, L}, skr[1] = {static_cast<uint64_t>(a.ld_cache) * 2};
  const uint64_t dv[3] = {vdim, H, L}, sv[2] = {vdim * 2, ldkv};
  int rc = encode_tensor_map_bf16(&m[0], a.q, 3, dq, sq, box3);
  if (rc == CTDK_OK) rc = encode_tensor_map_bf16(&m[1], a.q + dp, 3, dqr, sq, box3);
  if (rc == CTDK_OK) rc = encode_tensor_map_bf16(&m[2], a.kv, 3, dk, sk, box3);
  if (rc == CTDK_OK) rc = encode_tensor_map_bf16(&m[3], a.cache + a.rot_col, 2, dkr, skr, box2);
  if (rc == CTDK_OK) rc = encode_tensor_map_bf16(&m[4], a.kv + a.col_v, 3, dv, sv, box3);
  if (rc != CTDK_OK) return rc;
  TcArgs t;
  t.gate = a.proj + a.col_g;
  t.ld_gate = a.ldp;
  t.out = a.out;
  t.ld_out = a.ld_out;
  t.rows = static_cast<int>(rows);
  t.first = static_cast<int>(first);
  t.H = a.H;
  t.dim = a.dim;
  t.rot_dim = a.rot_dim;
  t.vdim = a.vdim;
  const int64_t items = (rows + TQ - 1) / TQ * a.H;
  CTDK_REQUIRE(items <= INT32_MAX / 2, "latent attention (tcgen05): too many tiles");
  t.n_items = static_cast<int>(items);
  t.scale_log2 = a.scale * kLog2e;
  t.status = device_status_word();
  if (t.status == nullptr) return fail(CTDK_ELAUNCH, "latent attention (tcgen05): no status word");
  if (a.dim <= 64) return a.vdim <= 64 ? launch<1, 1>(m, t, s) : launch<1, 2>(m, t, s);
  return a.vdim <= 64 ? launch<2, 1>(m, t, s) : launch<2, 2>(m, t, s);
}

}  // namespace hybrid
}  // namespace ctdk
