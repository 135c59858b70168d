// The parallel arrangement of the layer-list family (design Detatar): every layer has one norm, a token
// shift in front of the mixer, and mixer and feed-forward side by side, each behind a gate of its own.
//
// State per sequence and layer: the last normed row and, for time mixing, the last mixer input (two slots,
// a position writes slot position mod 2); for latent attention one row per position (latent and rotated key
// part); for time mixing the fp32 state. A layer that uses another's weights has all of this for itself.
// The residual is not updated behind a sublayer but by the next norm, which reads both sublayers' results
// and their gates.
#include <algorithm>

#include "hybrid_decoder.h"
#include "moe_route.cuh"

namespace ctdk {

int gemm_bf16_out16(const void* A, int64_t lda, const void* B, int64_t ldb, __nv_bfloat16* C, int64_t ldc, int64_t M, int N, int K, int up_row,
                    const int32_t* tiles, int max_tiles, int64_t n_pitch, int groups, cudaStream_t stream);

namespace hybrid {

template <typename T>
int HybridDecoder<T>::carve_parallel(Bump& b) {
  const int64_t R = max_portion, W = m.width, n_layers = static_cast<int64_t>(m.layers.size());
  const bool exact = m.dtype == CTDK_DTYPE_F32;
  int64_t n_in = 8, n_side = 8, heads_out = 8, low = 8, q_up_n = 0, q_rot_n = 0, kv_n = 0, act_n = 8, dz_n = 0, o_n = 0, parts = 0, abs_n = 0;
  int64_t low_w = 8, chunk_n = 0, decay_n = 0, choices = 0, counts = 0, tiles = 0, slots = 0, gu_n = 0, ea_n = 0, tegu_n = 0;
  bool mix = false, shared = false;
  bufs.assign(m.layers.size(), {});
  ropes.clear();
  for (size_t l = 0; l < m.layers.size(); ++l) {
    const Layer& L = m.layers[l];
    const Branch& br = L.branches[0];
    BranchBuffers bb;
    n_in = std::max<int64_t>(n_in, L.n_in);
    n_side = std::max<int64_t>(n_side, L.n_side);
    const int64_t out_n = static_cast<int64_t>(br.heads) * br.vdim;
    heads_out = std::max<int64_t>(heads_out, pad8(out_n));
    if (br.kind == BranchKind::kLatent) {
      bb.n_latent_rot = pad8(br.kv_rank);
      bb.ld_latent = bb.n_latent_rot + pad8(br.rot_dim);
      bb.latent = b.bytes(max_seq * bb.ld_latent * static_cast<int64_t>(sizeof(T)));
      low = std::max<int64_t>(low, br.ld_uq);
      q_up_n = std::max<int64_t>(q_up_n, pad8(static_cast<int64_t>(br.heads) * (br.dim + br.rot_dim)));
      q_rot_n = std::max<int64_t>(q_rot_n, static_cast<int64_t>(br.heads) * latent_q_pitch(br.dim, br.rot_dim));
      kv_n = std::max<int64_t>(kv_n, br.n_ukv);
      parts = std::max<int64_t>(parts, static_cast<int64_t>(br.heads) * kLatentSplits * (bb.n_latent_rot + kAttnStats4));
      abs_n = std::max<int64_t>(abs_n, br.heads * bb.ld_latent);
      for (size_t i = 0; i < ropes.size() && bb.rope < 0; ++i)
        if (ropes[i].spec == br.rope) bb.rope = static_cast<int>(i);
      if (bb.rope < 0) {
        RopeTable rt;
        rt.spec = br.rope;
        rt.rows = max_seq;
        rt.table = static_cast<float2*>(b.bytes(static_cast<int64_t>(max_seq) * (br.rope.dims / 2) * 8));
        rt.freqs = static_cast<double*>(b.bytes(br.rope.dims / 2 * 8));
        bb.rope = static_cast<int>(ropes.size());
        ropes.push_back(rt);
      }
    } else {
      mix = true;
      bb.state = b.floats(static_cast<int64_t>(br.heads) * br.dim * br.vdim);
      dz_n = std::max<int64_t>(dz_n, pad8(out_n));
      o_n = std::max<int64_t>(o_n, out_n);
      low_w = std::max<int64_t>(low_w, br.ld_w2);
      if (chunked_wkv(br)) {
        const int64_t tiles_n = (R + kWkvChunk - 1) / kWkvChunk * br.heads, d = wkv_tile(br.dim);
        chunk_n = std::max(chunk_n, tiles_n * d * d);
        decay_n = std::max(decay_n, tiles_n * d);
      }
    }
    bufs[l].push_back(bb);
    if (L.ffn == FeedForward::kGeluGlu) act_n = std::max<int64_t>(act_n, L.ffp);
    if (L.ffn == FeedForward::kMoe) {
      const Moe& e = L.moe;
      shared = shared || e.sff > 0;
      act_n = std::max<int64_t>(act_n, e.sffp);
      choices = std::max<int64_t>(choices, e.top);
      counts = std::max<int64_t>(counts, 2 * e.experts);
      const int64_t mt = moe_max_tiles(R, e.experts, e.top);
      tiles = std::max<int64_t>(tiles, mt + 2);
      slots = std::max<int64_t>(slots, mt * kMoeTile);
      gu_n = std::max<int64_t>(gu_n, mt * kMoeTile * 2 * e.effp);
      ea_n = std::max<int64_t>(ea_n, mt * kMoeTile * e.effp);
      tegu_n = std::max<int64_t>(tegu_n, static_cast<int64_t>(e.top) * 2 * e.effp);
    }
  }
  auto typed = [&](int64_t n) { return static_cast<T*>(b.bytes(n * static_cast<int64_t>(sizeof(T)))); };
  auto ints = [&](int64_t n) { return static_cast<int32_t*>(b.bytes(n * 4)); };
  shift_state = b.floats(n_layers * 4 * W);
  shift_next = b.floats(n_layers * 2 * W);
  x = b.floats(R * W);
  x2 = b.floats(R * W);
  h = typed(R * m.ldw);
  shifted = typed(R * m.ldw);
  mixes = typed(mix ? Branch::kMixes * R * m.ldw : 0);
  proj = b.floats(R * n_in);
  side = b.floats(R * n_side);
  y1 = b.floats(R * W);
  y2 = b.floats(R * W);
  mixed = typed(R * heads_out);
  o32 = b.floats(R * o_n);
  dz = b.floats(R * dz_n);
  low_a = typed(R * low_w);
  chunk_state = b.floats(chunk_n);
  cdecay = b.floats(decay_n);
  low_q = typed(R * low);
  q_up = b.floats(R * q_up_n);
  q_rot = typed(R * q_rot_n);
  kv_heads = typed(max_seq * kv_n);
  act = typed(R * act_n);
  moe_index = ints(R * choices);
  moe_slot = ints(R * choices);
  moe_weight = b.floats(R * choices);
  moe_count = ints(counts);
  moe_tiles = ints(tiles);
  expert_in = typed(slots * m.ldw);
  expert_gu = b.floats(exact ? gu_n : 0);
  expert_act = typed(ea_n);
  expert_out = typed(slots * m.ldw);
  shared_out = b.floats(shared ? R * W : 0);
  want_dev = ints(R);

  tx[0] = b.floats(W);
  tx[1] = b.floats(W);
  th = b.floats(W);
  tproj = b.floats(n_in);
  tside = b.floats(2 * n_side);
  tside_pitch = n_side;
  tq = b.floats(q_up_n);
  tq_abs = b.floats(abs_n);
  tegu = b.floats(tegu_n);
  tout[0] = b.floats(heads_out);
  ty1 = b.floats(W);
  ty2 = b.floats(W);
  tpart = b.floats(parts);
  sync_words = kTokenSyncWords;
  sync = static_cast<unsigned int*>(b.bytes(sync_words * 4));
  phases_dev = static_cast<TokenPhase*>(b.bytes((n_layers * 6 + 1) * static_cast<int64_t>(sizeof(TokenPhase))));
  logits = b.floats(vocab);
  cur_token = static_cast<int64_t*>(b.bytes(16));
  counters = static_cast<int*>(b.bytes(64));
  return CTDK_OK;
}

// The phases of one token: [norm + all projections of the layer] | latent attention: [queries] | [queries
// against the cache rows] | [ranges of the cache] | [merge + values], time mixing: [state] | [output
// projection]; the feed-forward rides along: experts' gate and up rows in the second phase, down rows in the
// third.
template <typename T>
int HybridDecoder<T>::build_parallel_phases() {
  phases.clear();
  stage_floats = 0;
  const int ldw = static_cast<int>(m.ldw), W = m.width;
  const int wpg = m.norm_groups >= kListWarps ? 1 : kListWarps / m.norm_groups;
  int cur = 0;
  auto need = [&](int64_t floats) { stage_floats = std::max<int>(stage_floats, static_cast<int>(floats)); };
  auto list = [&] {
    TokenPhase p{};
    p.stage = kStageList;
    p.prefetch = -1;
    return p;
  };
  auto add_op = [&](TokenPhase& p, int kind, int64_t at, int64_t n, int64_t ld, const float* src, const float* src2 = nullptr,
                    const float* w = nullptr) {
    p.op[p.n_ops++] = StageOp{kind, static_cast<int>(at), static_cast<int>(n), static_cast<int>(ld), src, src2, w};
    need(at + (kind == kOpRoute ? ld + n + route_scratch(static_cast<int>(n), p.route_groups) : std::max(n, ld)));
  };
  auto add_gemv = [&](TokenPhase& p, const T* w, float* y, int64_t rows, int64_t K, int64_t in) -> TokenGemv& {
    TokenGemv g{};
    g.W = w;
    g.y = y;
    g.rows = static_cast<int>(rows);
    g.K = static_cast<int>(K);
    g.in = static_cast<int>(in);
    p.gemv[p.n_gemv] = g;
    return p.gemv[p.n_gemv++];
  };
  auto norm_phase = [&](int64_t w, size_t l) {   // l: the layer in front of which this norm stands
    TokenPhase p = list();
    p.first_token = l == 0 ? 1 : 0;
    TokenShift& f = p.shift;
    f.groups = m.norm_groups;
    f.wpg = wpg;
    f.vec = W % (4 * m.norm_groups) == 0 ? 1 : 0;
    f.ld = ldw;
    f.w = vec(w);
    if (l > 0) {
      const Layer& B = m.layers[l - 1];
      const float* z = tside + ((l - 1) & 1) * tside_pitch;
      f.x = tx[cur];
      f.y1 = ty1;
      f.z1 = z + B.col_rg1;
      f.b1 = vec(B.b_rg1);
      if (B.ffn != FeedForward::kNone) {
        f.y2 = ty2;
        f.z2 = z + B.col_rg2;
        f.b2 = vec(B.b_rg2);
      }
      cur ^= 1;
    }
    p.op[p.n_ops++] = StageOp{kOpShiftNorm, 0, W, ldw, nullptr, nullptr, nullptr};
    return p;
  };
  for (size_t l = 0; l < m.layers.size(); ++l) {
    const Layer& L = m.layers[l];
    const Branch& br = L.branches[0];
    const BranchBuffers& bb = bufs[l][0];
    const Moe& e = L.moe;
    const bool moe = L.ffn == FeedForward::kMoe, latent = br.kind == BranchKind::kLatent;
    float* zs = tside + (l & 1) * tside_pitch;

    TokenPhase p = norm_phase(L.norm1, l);
    TokenShift& f = p.shift;
    f.shift = vec(L.shift);
    f.x_out = tx[cur];
    f.h_out = th;
    f.state = shift_state + static_cast<int64_t>(l) * 4 * W;
    f.n_mix = latent ? 0 : Branch::kMixes;
    f.red = (2 + f.n_mix) * ldw;
    need(f.red + m.norm_groups * wpg);
    if (latent) {
      add_gemv(p, at<T>(L.w_in), tproj, L.n_in, ldw, ldw);
    } else {
      const int64_t n = static_cast<int64_t>(br.heads) * br.dim;
      for (int i = 0; i < Branch::kMixes; ++i) {
        f.mu[i] = vec(br.mu[i]);
        add_gemv(p, at<T>(L.w_in) + static_cast<int64_t>(br.col_mix[i]) * ldw, tproj + br.col_mix[i], i < 4 ? n : br.rank_w, ldw, (2 + i) * ldw);
      }
    }
    add_gemv(p, at<T>(L.w_side), zs, L.n_side, ldw, 0);
    phases.push_back(p);

    TokenBranch t{};
    t.H = br.heads;
    t.G = br.kv_heads;
    t.dim = br.dim;
    t.vdim = br.vdim;
    t.col_k = br.col_k;
    t.col_g = br.col_g;
    t.out = tout[0];
    if (latent) {
      t.table = ropes[bb.rope].table;
      t.scale = br.scale;
      t.cache = bb.latent;
      t.part = tpart;
      t.rot_dim = br.rot_dim;
      t.kv_rank = br.kv_rank;
      t.rot_col = static_cast<int>(bb.n_latent_rot);
      t.ld_cache = static_cast<int>(bb.ld_latent);
      t.ld_ukv = static_cast<int>(br.ld_ukv);
      t.row_uv = br.row_uv;
      t.w_ukv = at<T>(br.w_ukv);
      t.kv_norm = vec(br.kv_norm);
      t.q_up = tq;
      t.q_abs = tq_abs;
      const int hb = sizeof(T) == 2 ? kLatentHeads : kLatentHeadsF32;
      t.blocks = (br.heads + hb - 1) / hb;
      t.splits = std::min(kLatentSplits, std::max(8, 2 * sm_count() / t.blocks));
    } else {
      t.kind = kTokWkv;
      t.items = br.heads * ((br.dim + 31) / 32);
      t.state = bb.state;
      t.col_r = br.col_mix[0];
      t.col_k = br.col_mix[1];
      t.col_v = br.col_mix[2];
      t.col_w1 = br.col_mix[4];
      t.rank_w = br.rank_w;
      t.w_w2 = at<T>(br.w_w2);
      t.w0 = vec(br.w0);
      t.bonus = vec(br.bonus);
    }
    // the choice, and h for the chosen experts
    auto expert_up = [&](TokenPhase& q, int64_t offset) {
      q.route_groups = e.groups;
      q.route_keep = e.keep;
      q.route_top = e.top;
      add_op(q, kOpRoute, offset, e.outputs(), ldw, zs + L.col_router, th, vec(e.correction));
      TokenGemv& g = add_gemv(q, at<T>(e.w_gu), tegu, static_cast<int64_t>(e.top) * 2 * e.effp, ldw, offset);
      g.mode = kGemvExpertUp;
      g.per = g.pitch = 2 * e.effp;
      g.top = e.top;
      g.experts = e.experts;
    };
    auto down = [&](TokenPhase& q, int64_t offset) {
      if (L.ffn == FeedForward::kGeluGlu) {
        add_op(q, kOpGelu, offset, L.ffp, L.ffp, zs + L.col_gu);
        add_gemv(q, at<T>(L.w_down), ty2, W, L.ld_down, offset);
        return;
      }
      if (!moe) return;
      q.route_top = e.top;
      add_op(q, kOpExperts, offset, e.effp, e.experts, tegu);
      const int64_t act_end = offset + static_cast<int64_t>(e.top) * e.effp;
      need(act_end);
      TokenGemv& g = add_gemv(q, at<T>(e.w_down), ty2, W, e.ld_down, offset);
      g.mode = kGemvExpertDown;
      g.pitch = pad8(W);
      g.top = e.top;
      g.experts = e.experts;
      g.h = th;
      if (e.sff > 0) {
        add_op(q, kOpShared, act_end, e.sffp, e.sffp, zs + L.col_gu, zs + L.col_sg);
        g.W2 = at<T>(e.w_sdown);
        g.K2 = static_cast<int>(e.ld_sdown);
        g.in2 = static_cast<int>(act_end);
      }
    };
    auto items = [&](TokenPhase& q, int kind, int n) {
      q.proj = tproj;
      q.n_branch = 1;
      q.br[0] = t;
      q.br[0].kind = kind;
      q.br[0].items = n;
    };
    const int64_t out_ld = br.ld_o;
    if (latent) {
      const int64_t esize = static_cast<int64_t>(sizeof(T));
      TokenPhase q = list();   // queries; the position's cache row
      items(q, kTokLatentKeys, 0);
      add_gemv(q, at<T>(br.w_uq), tq, static_cast<int64_t>(br.heads) * (br.dim + br.rot_dim), br.ld_uq, 0);
      if (moe) expert_up(q, br.ld_uq);   // one warp chooses while the others go on
      add_op(q, kOpRmsNorm, 0, br.q_rank, br.ld_uq, tproj + br.col_q, nullptr, vec(br.q_norm));
      add_op(q, kOpLatentStore, 0, 0, 0, nullptr);
      phases.push_back(q);

      const int key_cols = 16 * (16 / static_cast<int>(sizeof(T)));
      TokenPhase k = list();   // queries against the cache rows
      items(k, kTokLatentKeys, br.heads * ((t.rot_col + key_cols - 1) / key_cols));
      down(k, 0);
      need(kListThreads / 16 * (key_cols + 1));
      k.extra = at<T>(br.w_ukv);
      k.extra_bytes = static_cast<int64_t>(br.row_uv) * br.ld_ukv * esize;
      phases.push_back(k);

      TokenPhase sc = list();
      items(sc, kTokLatentScan, t.blocks * t.splits);
      const int64_t slices = (t.ld_cache + 15) / 16 * 16 + 8;   // bfloat16 pitch
      const int64_t tile = sizeof(T) == 2 ? kLatentKeys * slices / 2 : 4 * kLatentKeys * (t.ld_cache / 4 | 1);
      const int64_t queries = sizeof(T) == 2 ? kLatentHeads * (slices + kLatentKeys + 8 + 8 * (kLatentKeys + 4) + 1)
                                             : kLatentHeadsF32 * (t.ld_cache + kLatentKeys + 1);
      sc.br[0].buffers = 4 * (queries + 2 * tile) <= 190 * 1024 ? 2 : 1;
      need(queries + sc.br[0].buffers * tile);
      phases.push_back(sc);

      TokenPhase v = list();
      items(v, kTokLatentOut, br.heads * ((br.vdim + kLatentOutRows - 1) / kLatentOutRows));
      need(t.rot_col * (1 + kLatentOutParts) + kLatentSplits);
      v.extra = at<T>(br.w_ukv) + static_cast<int64_t>(br.row_uv) * br.ld_ukv;
      v.extra_bytes = static_cast<int64_t>(br.heads) * br.vdim * br.ld_ukv * esize;
      phases.push_back(v);

      TokenPhase o = list();
      add_op(o, kOpCopy, 0, static_cast<int64_t>(br.heads) * br.vdim, out_ld, tout[0]);
      add_gemv(o, at<T>(br.w_o), ty1, W, out_ld, 0);
      phases.push_back(o);
    } else {
      TokenPhase q = list();
      items(q, kTokWkv, t.items);
      need(br.ld_w2 + 4 * br.dim + kListThreads);
      if (moe) expert_up(q, 0);
      phases.push_back(q);

      TokenPhase o = list();
      items(o, kTokWkv, 0);
      add_op(o, kOpHeadNorm, 0, static_cast<int64_t>(br.heads) * br.dim, out_ld, tout[0], tproj + br.col_mix[3], vec(br.w_norm));
      add_gemv(o, at<T>(br.w_o), ty1, W, out_ld, 0);
      down(o, out_ld);
      phases.push_back(o);
    }
  }
  TokenPhase hd = norm_phase(m.final_norm, m.layers.size());
  hd.shift.red = ldw;
  need(ldw + m.norm_groups * wpg);
  hd.is_head = 1;
  add_gemv(hd, at<T>(m.head), logits, vocab, ldw, 0);
  phases.push_back(hd);
  return finish_phases();
}

template <>
int HybridDecoder<float>::kv_rows(const float* cache, const float* w, int64_t rows, int64_t n, int64_t K, int64_t lda, int64_t ldw, cudaStream_t s) {
  return gemm_rows(cache, w, kv_heads, rows, n, K, lda, ldw, n, s);
}
template <>
int HybridDecoder<__nv_bfloat16>::kv_rows(const __nv_bfloat16* cache, const __nv_bfloat16* w, int64_t rows, int64_t n, int64_t K, int64_t lda,
                                          int64_t ldw, cudaStream_t s) {
  return gemm_bf16_out16(cache, lda, w, ldw, kv_heads, n, rows, static_cast<int>(n), static_cast<int>(K), 0, nullptr, 0, 0, 1, s);
}
template <>
int HybridDecoder<float>::latent_attention(const LatentArgs<float>& a, int64_t pos, int64_t n, cudaStream_t s) {
  return latent_attention_fp32(a, pos, n, s);
}
template <>
int HybridDecoder<__nv_bfloat16>::latent_attention(const LatentArgs<__nv_bfloat16>& a, int64_t pos, int64_t n, cudaStream_t s) {
  if (latent_tcgen05_ok(a.dim, a.rot_dim, a.vdim)) return latent_attention_tcgen05(a, pos, n, s);
  return latent_attention_fp32(a, pos, n, s);
}

template <typename T>
int HybridDecoder<T>::mixer_latent(const Layer& L, const BranchBuffers& bb, int64_t n, int64_t pos, cudaStream_t s) {
  const Branch& b = L.branches[0];
  const int64_t ldp = L.n_in;
  DTRY(gemm_rows(shifted, at<T>(L.w_in), proj, n, ldp, m.width, m.ldw, m.ldw, ldp, s));
  LatentArgs<T> a;
  a.proj = proj;
  a.ldp = ldp;
  a.col_q = b.col_q;
  a.col_k = b.col_k;
  a.col_g = b.col_g;
  a.H = b.heads;
  a.dim = b.dim;
  a.rot_dim = b.rot_dim;
  a.vdim = b.vdim;
  a.kv_rank = b.kv_rank;
  a.q_rank = b.q_rank;
  a.eps = m.eps;
  a.scale = b.scale;
  a.q_norm = vec(b.q_norm);
  a.kv_norm = vec(b.kv_norm);
  a.table = ropes[bb.rope].table;
  a.cache = static_cast<T*>(bb.latent);
  a.ld_cache = bb.ld_latent;
  a.rot_col = static_cast<int>(bb.n_latent_rot);
  a.low_q = low_q;
  a.ld_low = b.ld_uq;
  a.q_up = q_up;
  a.ld_up = pad8(static_cast<int64_t>(b.heads) * (b.dim + b.rot_dim));
  a.q = q_rot;
  a.kv = kv_heads;
  a.ld_kv = b.n_ukv;
  a.col_v = b.row_uv;
  a.out = mixed;
  a.ld_out = b.ld_o;
  DTRY(latent_prep(a, pos, n, s));
  DTRY(gemm_rows(low_q, at<T>(b.w_uq), q_up, n, a.ld_up, b.q_rank, b.ld_uq, b.ld_uq, a.ld_up, s));
  DTRY(latent_rotate(a, pos, n, s));
  // keys and values of every position so far, out of the cached latents
  DTRY(kv_rows(a.cache, at<T>(b.w_ukv), pos + n, b.n_ukv, b.kv_rank, a.ld_cache, b.ld_ukv, s));
  DTRY(latent_attention(a, pos, n, s));
  return gemm_rows(mixed, at<T>(b.w_o), y1, n, m.width, static_cast<int64_t>(b.heads) * b.vdim, b.ld_o, b.ld_o, m.width, s);
}

template <typename T>
int HybridDecoder<T>::mixer_wkv(const Layer& L, const BranchBuffers& bb, int64_t n, int64_t pos, cudaStream_t s) {
  const Branch& b = L.branches[0];
  const int64_t ldp = L.n_in;
  const int64_t cols = static_cast<int64_t>(b.heads) * b.dim, ldz = pad8(cols);
  for (int i = 0; i < Branch::kMixes; ++i)
    DTRY(gemm_rows(mixes + i * n * m.ldw, at<T>(L.w_in) + static_cast<int64_t>(b.col_mix[i]) * m.ldw, proj + b.col_mix[i], n,
                   i < 4 ? pad8(cols) : pad8(b.rank_w), m.width, m.ldw, m.ldw, ldp, s));
  DTRY(tanh_rows(proj + b.col_mix[4], ldp, low_a, b.ld_w2, n, b.rank_w, s));
  DTRY(gemm_rows(low_a, at<T>(b.w_w2), dz, n, ldz, b.rank_w, b.ld_w2, b.ld_w2, ldz, s));
  if (chunked_wkv(b) && n >= kChunkedRows) {
    WkvArgs c;
    c.r = proj + b.col_mix[0];
    c.k = proj + b.col_mix[1];
    c.v = proj + b.col_mix[2];
    c.gate = proj + b.col_mix[3];
    c.ldp = ldp;
    c.z = dz;
    c.ldz = ldz;
    c.w0 = vec(b.w0);
    c.bonus = vec(b.bonus);
    c.w_norm = vec(b.w_norm);
    c.state = bb.state;
    c.chunk_state = chunk_state;
    c.decay = cdecay;
    c.out = reinterpret_cast<__nv_bfloat16*>(mixed);   // chunked_wkv: the model's type
    c.ld_out = b.ld_o;
    c.H = b.heads;
    c.dim = b.dim;
    c.eps = m.eps;
    c.rows = n;
    c.resume = pos > 0;
    DTRY(wkv_chunked(c, s));
    return gemm_rows(mixed, at<T>(b.w_o), y1, n, m.width, cols, b.ld_o, b.ld_o, m.width, s);
  }
  ScanArgs a;
  a.q = proj + b.col_mix[0];
  a.k = proj + b.col_mix[1];
  a.v = proj + b.col_mix[2];
  a.ldq = a.ldk = a.ldv = ldp;
  a.z = dz;
  a.ldz = ldz;
  a.w0 = vec(b.w0);
  a.bonus = vec(b.bonus);
  a.state = bb.state;
  a.out = o32;
  a.H = a.G = b.heads;
  a.dim = a.vdim = b.dim;
  a.rows = n;
  a.resume = pos > 0;
  DTRY(recurrent_scan(a, Recurrence::kWkv, s));
  DTRY(silu_head_norm_rows(o32, vec(b.w_norm), proj + b.col_mix[3], ldp, mixed, b.ld_o, n, b.heads, b.dim, m.eps, s));
  return gemm_rows(mixed, at<T>(b.w_o), y1, n, m.width, cols, b.ld_o, b.ld_o, m.width, s);
}

// y2 = feed-forward of h; side holds what the layer's unshifted projections gave.
template <typename T>
int HybridDecoder<T>::feed_forward_rows(const Layer& L, int64_t n, cudaStream_t s) {
  if (L.ffn == FeedForward::kGeluGlu) {
    DTRY(glu_rows(side + L.col_gu, L.n_side, act, L.ffp, n, L.ffp, Glu::kGelu, nullptr, s));
    return gemm_rows(act, at<T>(L.w_down), y2, n, m.width, L.ff, L.ffp, L.ld_down, m.width, s);
  }
  if (L.ffn != FeedForward::kMoe) return CTDK_OK;
  const Moe& e = L.moe;
  const float* shared = nullptr;
  if (e.sff > 0) {
    DTRY(glu_rows(side + L.col_gu, L.n_side, act, e.sffp, n, e.sffp, Glu::kSilu, nullptr, s));
    DTRY(gemm_rows(act, at<T>(e.w_sdown), shared_out, n, m.width, e.sff, e.sffp, e.ld_sdown, m.width, s));
    shared = shared_out;
  }
  MoeArgs a;
  a.z = side + L.col_router;
  a.ldz = L.n_side;
  a.correction = vec(e.correction);
  a.experts = e.experts;
  a.outputs = e.outputs();
  a.top = e.top;
  a.groups = e.groups;
  a.keep = e.keep;
  a.index = moe_index;
  a.slot = moe_slot;
  a.weight = moe_weight;
  a.count = moe_count;
  a.tiles = moe_tiles;
  a.max_tiles = static_cast<int>(moe_max_tiles(n, e.experts, e.top));
  DTRY(moe_route(a, n, s));
  DTRY(moe_gather(a, h, m.ldw, expert_in, m.width, n, s));
  DTRY(experts_up(a, expert_in, m.ldw, at<T>(e.w_gu), m.ldw, m.width, e.effp, expert_act, expert_gu, s));
  DTRY(experts_down(a, expert_act, e.effp, at<T>(e.w_down), e.ld_down, pad8(m.width), m.width, e.eff, expert_out, m.ldw, s));
  return moe_combine(a, expert_out, m.ldw, h, m.ldw, side + L.col_sg, L.n_side, shared, y2, m.width, n, s);
}

// n <= max_portion rows at positions pos ..; `done` rows of the caller's portion came before.
template <typename T>
int HybridDecoder<T>::run_parallel_rows(const int64_t* ids, int64_t n, int64_t pos, int64_t done, const int32_t* want, int64_t n_want,
                                        float* want_logits, bool last, cudaStream_t s) {
  const int W = m.width, n_layers = static_cast<int>(m.layers.size());
  float *x_now = x, *x_next = x2;
  ShiftNormArgs<T> na;   // what the next norm adds to the residual
  na.width = W;
  na.groups = m.norm_groups;
  na.eps = m.eps;
  na.scale = m.embed_scale;
  na.ids = ids;
  na.embed = at<T>(m.embed);
  na.ld_embed = m.ldw;
  na.h = h;
  na.shifted = shifted;
  na.mix = mixes;
  na.mix_stride = n * m.ldw;
  na.ld_h = m.ldw;
  for (int l = 0; l < n_layers; ++l) {
    const Layer& L = m.layers[l];
    const Branch& br = L.branches[0];
    const float* state = shift_state + (static_cast<int64_t>(l) * 2 + ((pos + 1) & 1)) * 2 * W;
    na.x = x_now;
    na.x_out = x_next;
    na.w = vec(L.norm1);
    na.shift = vec(L.shift);
    na.n_mix = br.kind == BranchKind::kWkv ? Branch::kMixes : 0;
    for (int i = 0; i < na.n_mix; ++i) na.mu[i] = vec(br.mu[i]);
    na.prev_h = pos > 0 ? state : nullptr;
    na.prev_m = pos > 0 ? state + W : nullptr;
    na.next_h = shift_next + static_cast<int64_t>(l) * 2 * W;
    na.next_m = na.next_h + W;
    DTRY(shift_norm_rows(na, n, s));
    if (layers_out != nullptr && l > 0 &&
        cudaMemcpyAsync(layers_out + (l - 1) * n * W, x_next, n * W * 4, cudaMemcpyDeviceToDevice, s) != cudaSuccess)
      return fail(CTDK_ELAUNCH, "hybrid decoder: copying the residual failed");
    std::swap(x_now, x_next);
    DTRY(gemm_rows(h, at<T>(L.w_side), side, n, L.n_side, W, m.ldw, m.ldw, L.n_side, s));
    if (br.kind == BranchKind::kLatent) DTRY(mixer_latent(L, bufs[l][0], n, pos, s));
    else DTRY(mixer_wkv(L, bufs[l][0], n, pos, s));
    DTRY(feed_forward_rows(L, n, s));
    na.ids = nullptr;
    na.y1 = y1;
    na.z1 = side + L.col_rg1;
    na.b1 = vec(L.b_rg1);
    na.y2 = L.ffn != FeedForward::kNone ? y2 : nullptr;
    na.z2 = side + L.col_rg2;
    na.b2 = L.ffn != FeedForward::kNone ? vec(L.b_rg2) : nullptr;
    na.ldz = L.n_side;
  }
  DTRY(commit_shift_state(shift_next, shift_state, n_layers, static_cast<int>((pos + n - 1) & 1), W, s));
  na.x = x_now;
  na.w = vec(m.final_norm);
  na.shift = nullptr;
  na.n_mix = 0;
  if (layers_out != nullptr) {   // the last layer's residual, which is otherwise only formed for the wanted rows
    na.x_out = layers_out + static_cast<int64_t>(n_layers - 1) * n * W;
    DTRY(shift_norm_rows(na, n, s));
  }
  na.x_out = nullptr;
  return run_head(n, done, want, n_want, want_logits, last, [&](const int32_t* gather, int64_t k) {
    ShiftNormArgs<T> fa = na;
    fa.gather = gather;
    return shift_norm_rows(fa, k, s);
  }, s);
}

#define INSTANTIATE(T)                                                                                                                   \
  template int HybridDecoder<T>::carve_parallel(Bump&);                                                                                  \
  template int HybridDecoder<T>::build_parallel_phases();                                                                                \
  template int HybridDecoder<T>::run_parallel_rows(const int64_t*, int64_t, int64_t, int64_t, const int32_t*, int64_t, float*, bool, \
                                                   cudaStream_t);
INSTANTIATE(float)
INSTANTIATE(__nv_bfloat16)

}  // namespace hybrid
}  // namespace ctdk
