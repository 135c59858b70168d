// Decoder of the layer-list family: caches and recurrent states, the prompt pass (portions of any
// size on the tensor-core products) and the phase list of the persistent token kernel. Request loop:
// decode_api.cu.
//
// State per sequence: for an attention branch the unrotated keys of the current chunk (they are the
// values too; slot = position mod chunk), for a recurrence its fp32 state, for a short convolution its
// last inputs (slot = position mod taps). Position 0 starts from nothing whatever these buffers hold,
// so a reset costs no device work.
#include <algorithm>
#include <cmath>
#include <new>
#include <vector>

#include "hybrid_decoder.h"

namespace ctdk {
namespace hybrid {

template <typename T>
int HybridDecoder<T>::carve(Bump& b) {
  if (m.arrangement == Arrangement::kParallel) return carve_parallel(b);
  const int64_t R = max_portion, W = m.width;
  int64_t n_in = 8, mix = 8, heads_out = 8, packed_n = 0, attn_n = 0, ff = 8, parts = 0, arrives = 0;
  int64_t ck_n = 0, cv_n = 0, cs_n = 0, cd_n = 0;
  int64_t chunk_n = 0, qk_tiles = 0, v_tiles = 0;
  int64_t qk = 0, dv_n = 0, dlog_n = 0, db_n = 0, rank = 8, rank_g = 8, gate_n = 0;
  bufs.assign(m.layers.size(), {});
  ropes.clear();
  for (size_t l = 0; l < m.layers.size(); ++l) {
    const Layer& L = m.layers[l];
    n_in = std::max<int64_t>(n_in, L.n_in);
    ff = std::max<int64_t>(ff, L.ffp);
    for (const Branch& br : L.branches) {
      BranchBuffers bb;
      const int64_t out_n = static_cast<int64_t>(br.heads) * br.vdim;
      heads_out = std::max(heads_out, out_n);
      mix = std::max<int64_t>(mix, pad8(out_n));
      if (br.kind == BranchKind::kAttention) {
        bb.chunk = br.chunk > 0 && br.chunk < max_seq ? br.chunk : max_seq;
        bb.cache = b.bytes(br.kv_heads * bb.chunk * br.dim * static_cast<int64_t>(sizeof(T)));
        const int Dp = padded_head(br.dim, tensor_core_attention(br));
        const int64_t rows = (bb.chunk - 1 + R + bb.chunk - 1) / bb.chunk * bb.chunk;
        packed_n = std::max(packed_n, rows * (br.heads + 2 * br.kv_heads) * Dp);
        attn_n = std::max(attn_n, rows * br.heads * Dp);
        parts = std::max<int64_t>(parts, static_cast<int64_t>(br.heads) * kAttnSplits * (br.dim + kAttnStats));
        arrives = std::max<int64_t>(arrives, br.kv_heads);
        for (size_t i = 0; i < ropes.size() && bb.rope < 0; ++i)
          if (ropes[i].spec == br.rope && ropes[i].rows >= bb.chunk) bb.rope = static_cast<int>(i);
        if (bb.rope < 0) {
          RopeTable rt;
          rt.spec = br.rope;
          rt.rows = bb.chunk;
          rt.table = static_cast<float2*>(b.bytes(bb.chunk * (br.rope.dims / 2) * 8));
          rt.freqs = static_cast<double*>(b.bytes(br.rope.dims / 2 * 8));
          bb.rope = static_cast<int>(ropes.size());
          ropes.push_back(rt);
        }
      } else {
        bb.state = b.floats(static_cast<int64_t>(br.heads) * br.dim * br.vdim);
        if (br.kind == BranchKind::kLightning) {
          bb.decay = b.floats(br.heads);
          bb.powers = b.floats(static_cast<int64_t>(br.heads) * (kLightningChunk + 1));
          if (chunked_lightning(br)) {
            const int64_t tiles = ((R + kLightningChunk - 1) / kLightningChunk) * br.heads;
            const int64_t dk = lightning_tile(br.dim), dv = lightning_tile(br.vdim);
            chunk_n = std::max(chunk_n, tiles * dk * dv);
            qk_tiles = std::max(qk_tiles, tiles * kLightningChunk * dk);
            v_tiles = std::max(v_tiles, tiles * kLightningChunk * dv);
          }
        } else {
          bb.ring = b.floats(static_cast<int64_t>(br.taps) * (2 * br.kv_heads * br.dim + out_n));
          qk = std::max<int64_t>(qk, static_cast<int64_t>(br.kv_heads) * br.dim);
          dv_n = std::max<int64_t>(dv_n, out_n);
          dlog_n = std::max<int64_t>(dlog_n, pad8(static_cast<int64_t>(br.heads) * br.dim));
          gate_n = std::max<int64_t>(gate_n, pad8(out_n));
          if (delta_chunked_ok(br.dim, br.vdim)) {
            const int64_t tiles = ((R + kDeltaChunk - 1) / kDeltaChunk) * br.heads;
            const int64_t tk = lightning_tile(br.dim), tv = lightning_tile(br.vdim);
            chunk_n = std::max(chunk_n, tiles * tk * tv);
            ck_n = std::max(ck_n, tiles * kDeltaChunk * tk);
            cv_n = std::max(cv_n, tiles * kDeltaChunk * tv);
            cs_n = std::max(cs_n, tiles * kDeltaChunk * kDeltaChunk);
            cd_n = std::max(cd_n, tiles * tk);
          }
          db_n = std::max<int64_t>(db_n, br.heads);
          rank = std::max<int64_t>(rank, pad8(br.rank_a));
          rank_g = std::max<int64_t>(rank_g, pad8(br.rank_g));
        }
      }
      bufs[l].push_back(bb);
    }
  }
  auto typed = [&](int64_t n) { return static_cast<T*>(b.bytes(n * static_cast<int64_t>(sizeof(T)))); };
  x = b.floats(R * W);
  h = typed(R * m.ldw);
  proj = b.floats(R * n_in);
  packed = b.floats(packed_n);
  attn_out = b.floats(attn_n);
  o32 = b.floats(R * heads_out);
  mixed = typed(R * mix);
  y1 = b.floats(R * W);
  y2 = b.floats(R * W);
  gu = b.floats(R * 2 * ff);
  act = typed(R * ff);
  dq = b.floats(R * qk);
  dk = b.floats(R * qk);
  dv = b.floats(R * dv_n);
  dlog = b.floats(R * dlog_n);
  dz = b.floats(R * dlog_n);
  dgate = b.floats(R * gate_n);
  dbeta = b.floats(R * db_n);
  low_a = typed(R * rank);
  low_g = typed(R * rank_g);
  chunk_state = b.floats(chunk_n);
  cw = b.floats(ck_n);
  ckh = b.floats(ck_n);
  cqt = b.floats(ck_n);
  cu = b.floats(cv_n);
  cus = b.floats(cv_n);
  cscores = b.floats(cs_n);
  cdecay = b.floats(cd_n);
  qb = static_cast<__nv_bfloat16*>(b.bytes(qk_tiles * 2));
  kb = static_cast<__nv_bfloat16*>(b.bytes(qk_tiles * 2));
  vb = static_cast<__nv_bfloat16*>(b.bytes(v_tiles * 2));
  want_dev = static_cast<int32_t*>(b.bytes(R * 4));

  tx[0] = b.floats(W);
  tx[1] = b.floats(W);
  tproj = b.floats(n_in);
  tout[0] = b.floats(heads_out);
  tout[1] = b.floats(heads_out);
  tgate = b.floats(heads_out);
  ty1 = b.floats(W);
  ty2 = b.floats(W);
  tgu = b.floats(2 * ff);
  tpart = b.floats(parts);
  sync_words = kTokenSyncWords + 2 * arrives;
  sync = static_cast<unsigned int*>(b.bytes(sync_words * 4));
  phases_dev = static_cast<TokenPhase*>(b.bytes(static_cast<int64_t>(m.layers.size() * 5 + 1) * sizeof(TokenPhase)));
  logits = b.floats(vocab);
  cur_token = static_cast<int64_t*>(b.bytes(16));
  counters = static_cast<int*>(b.bytes(64));
  return CTDK_OK;
}

// The phases of one token (see hybrid_token.cu).
template <typename T>
int HybridDecoder<T>::build_phases() {
  if (m.arrangement == Arrangement::kParallel) return build_parallel_phases();
  phases.clear();
  stage_floats = static_cast<int>(m.ldw);
  int cur = 0;                       // which of tx[] holds the residual
  const float* pend_y = nullptr;     // sublayer output not yet added to the residual
  const float *pend_y2 = nullptr, *w_y = nullptr, *w_y2 = nullptr, *w_post = nullptr;
  auto product = [&](int stage) {
    TokenPhase p{};
    p.stage = stage;
    p.prefetch = -1;
    return p;
  };
  auto norm_phase = [&](const float* w_pre, bool store) {
    TokenPhase p = product(kStageNorm);
    p.first_token = phases.empty() ? 1 : 0;
    p.w_pre = w_pre;
    if (!p.first_token) {
      p.x = tx[cur];
      p.y = pend_y;
      p.y2 = pend_y2;
      p.w_y = w_y;
      p.w_y2 = w_y2;
      p.w_post = w_post;
      cur ^= 1;
    }
    p.x_out = store ? tx[cur] : nullptr;
    return p;
  };
  for (size_t l = 0; l < m.layers.size(); ++l) {
    const Layer& L = m.layers[l];
    TokenPhase p = norm_phase(vec(L.norm1), true);
    p.n_gemv = 1;
    p.gemv[0] = TokenGemv{at<T>(L.w_in), tproj, L.n_in, static_cast<int>(m.ldw), 0};
    phases.push_back(p);

    TokenPhase mx{};
    mx.is_mix = 1;
    mx.prefetch = -1;
    mx.proj = tproj;
    mx.n_branch = static_cast<int>(L.branches.size());
    TokenPhase o = product(kStageMixed);
    o.proj = tproj;
    o.n_branch = mx.n_branch;
    o.n_gemv = mx.n_branch;
    int offset = 0;
    for (int b = 0; b < mx.n_branch; ++b) {
      const Branch& br = L.branches[b];
      const BranchBuffers& bb = bufs[l][b];
      TokenBranch t{};
      t.H = br.heads;
      t.G = br.kv_heads;
      t.dim = br.dim;
      t.vdim = br.vdim;
      t.col_q = br.col_q;
      t.col_k = br.col_k;
      t.col_v = br.col_v;
      t.col_g = br.col_g;
      t.out = tout[b];
      t.stage_at = offset;
      const int column_blocks = (br.vdim + 31) / 32;
      if (br.kind == BranchKind::kAttention) {
        t.kind = kTokAttention;
        t.items = br.kv_heads * kAttnSplits;
        t.b_q = vec(br.b_q);
        t.b_k = vec(br.b_k);
        t.table = ropes[bb.rope].table;
        t.rot_pairs = br.rope.dims / 2;
        t.chunk = static_cast<int>(bb.chunk);
        t.scale = br.scale;
        t.cache = bb.cache;
        t.part = tpart;
        t.arrive = sync + kTokenSyncWords + b * ((sync_words - kTokenSyncWords) / 2);
      } else if (br.kind == BranchKind::kLightning) {
        t.kind = kTokLightning;
        t.items = br.heads * column_blocks;
        t.decay = bb.decay;
        t.state = bb.state;
        t.w_norm = vec(br.w_norm);
      } else {
        t.kind = kTokDelta;
        t.items = br.heads * column_blocks;
        t.state = bb.state;
        t.w_norm = vec(br.w_norm);
        t.taps = br.taps;
        t.col_b = br.col_b;
        t.col_a1 = br.col_a1;
        t.col_g1 = br.col_g1;
        t.rank_a = br.rank_a;
        t.rank_g = br.rank_g;
        t.conv_q = vec(br.conv_q);
        t.conv_k = vec(br.conv_k);
        t.conv_v = vec(br.conv_v);
        t.a_log = vec(br.a_log);
        t.dt_bias = vec(br.dt_bias);
        t.w_a2 = at<T>(br.w_a2);
        t.w_g2 = at<T>(br.w_g2);
        t.ring = bb.ring;
        t.gate = tgate;
      }
      o.gemv[b] = TokenGemv{at<T>(br.w_o), b == 0 ? ty1 : ty2, m.width, static_cast<int>(br.ld_o), offset};
      offset += static_cast<int>(br.ld_o);
      mx.br[b] = t;
      o.br[b] = t;
    }
    stage_floats = std::max(stage_floats, offset);
    phases.push_back(mx);
    phases.push_back(o);
    pend_y = ty1;
    const bool two = mx.n_branch == 2;
    pend_y2 = two ? ty2 : nullptr;
    w_y = two ? vec(L.branches[0].w_out) : nullptr;
    w_y2 = two ? vec(L.branches[1].w_out) : nullptr;
    w_post = vec(L.norm1b);
    if (L.ff > 0) {
      TokenPhase g = norm_phase(vec(L.norm2), true);
      g.n_gemv = 1;
      g.gemv[0] = TokenGemv{at<T>(L.w_gu), tgu, 2 * L.ffp, static_cast<int>(m.ldw), 0};
      phases.push_back(g);
      TokenPhase d = product(kStageGlu);
      d.gu = tgu;
      d.ffp = L.ffp;
      d.limit = L.limit;
      d.n_gemv = 1;
      d.gemv[0] = TokenGemv{at<T>(L.w_down), ty1, m.width, static_cast<int>(L.ld_down), 0};
      phases.push_back(d);
      stage_floats = std::max(stage_floats, L.ffp);
      pend_y = ty1;
      pend_y2 = w_y = w_y2 = nullptr;
      w_post = vec(L.norm2b);
    }
  }
  TokenPhase hd = norm_phase(vec(m.final_norm), false);
  hd.is_head = 1;
  hd.n_gemv = 1;
  hd.gemv[0] = TokenGemv{at<T>(m.head), logits, vocab, static_cast<int>(m.ldw), 0};
  phases.push_back(hd);

  return finish_phases();
}

// Prefetch order, shared memory, warps per row.
template <typename T>
int HybridDecoder<T>::finish_phases() {
  // every phase asks for the weights of one coming product, the mix phases run the queue one ahead
  const int n = static_cast<int>(phases.size());
  int next = 1;
  for (int i = 0; i < n; ++i) {
    next = std::max(next, i + 1);
    while (next < n && (phases[next].is_mix || (phases[next].n_gemv == 0 && phases[next].extra == nullptr))) ++next;
    if (next < n && next - i <= 3) phases[i].prefetch = next++;
  }
  token_smem = token_smem_bytes(stage_floats, phases.data(), n);
  CTDK_REQUIRE(token_smem <= 200 * 1024, "hybrid decoder: the token pass needs %zu bytes of shared memory", token_smem);
  int rc = token_grid<T>(token_smem, m.arrangement == Arrangement::kParallel, &token_ctas);
  if (rc != CTDK_OK) return rc;
  for (TokenPhase& p : phases) {
    if (p.is_mix) continue;
    int rows = 0, K = 0;
    for (int i = 0; i < p.n_gemv; ++i) {
      rows += p.gemv[i].rows;
      K = std::max(K, p.gemv[i].K);
    }
    int wpr = 1;
    while (wpr < 8 && static_cast<int64_t>(rows) * wpr * 2 <= static_cast<int64_t>(token_ctas) * 8 &&
           K * static_cast<int>(sizeof(T)) / 16 >= 64 * wpr)
      wpr *= 2;
    p.wpr = wpr;
  }
  return CTDK_OK;
}

// Constant tables: phases, decays, rotations. Synchronises (creation time only).
template <typename T>
int HybridDecoder<T>::upload(cudaStream_t s) {
  auto copy = [&](void* dst, const void* src, size_t n) { return cudaMemcpyAsync(dst, src, n, cudaMemcpyHostToDevice, s) == cudaSuccess; };
  std::vector<std::vector<float>> powers;
  bool ok = copy(phases_dev, phases.data(), phases.size() * sizeof(TokenPhase));
  for (size_t l = 0; l < m.layers.size(); ++l)
    for (size_t b = 0; b < bufs[l].size(); ++b)
      if (bufs[l][b].decay != nullptr) {
        const std::vector<float>& d = m.layers[l].branches[b].decay;
        powers.emplace_back();
        for (const float x : d)
          for (int i = 0; i <= kLightningChunk; ++i) powers.back().push_back(static_cast<float>(std::pow(static_cast<double>(x), i)));
        ok = ok && copy(bufs[l][b].powers, powers.back().data(), powers.back().size() * 4);
        ok = ok && copy(bufs[l][b].decay, d.data(), d.size() * 4);
      }
  std::vector<std::vector<double>> freqs;
  for (RopeTable& r : ropes) {
    std::vector<double> f(r.spec.dims / 2);
    for (size_t i = 0; i < f.size(); ++i) f[i] = r.spec.frequency(static_cast<int>(i));
    freqs.push_back(f);
    ok = ok && copy(r.freqs, freqs.back().data(), f.size() * 8);
    DTRY(rope_table_f64(r.table, r.rows, r.freqs, r.spec.dims / 2, s));
  }
  ok = ok && cudaMemsetAsync(counters, 0, 64, s) == cudaSuccess && cudaStreamSynchronize(s) == cudaSuccess;
  return ok ? CTDK_OK : fail(CTDK_ELAUNCH, "hybrid decoder: set-up copies failed");
}

template <typename T>
int HybridDecoder<T>::mixer_attention(const Branch& b, const BranchBuffers& bb, int64_t n, int64_t pos, float* y, int64_t ldp,
                                      cudaStream_t s) {
  AttnArgs<T> a;
  a.proj = proj;
  a.ldp = ldp;
  a.col_q = b.col_q;
  a.col_k = b.col_k;
  a.col_g = b.col_g;
  a.b_q = vec(b.b_q);
  a.b_k = vec(b.b_k);
  a.H = b.heads;
  a.G = b.kv_heads;
  a.dim = b.dim;
  const bool tc = tensor_core_attention(b);
  a.Dp = padded_head(b.dim, tc);
  a.rot_pairs = b.rope.dims / 2;
  a.chunk = bb.chunk;
  a.table = ropes[bb.rope].table;
  a.cache = static_cast<T*>(bb.cache);
  a.packed = packed;
  a.out = attn_out;
  const int64_t first = pos % bb.chunk, rows = first + n;
  DTRY(attn_pack(a, first, rows, s));
  DTRY(attn_store(a, first, rows, s));
  if (tc) DTRY(attn_chunked_tcgen05(packed, attn_out, rows, first, bb.chunk, b.heads, b.kv_heads, a.Dp, b.scale, s));
  else DTRY(attn_chunked_fp32(packed, attn_out, first, rows, bb.chunk, b.heads, b.kv_heads, b.dim, a.Dp, b.scale, s));
  DTRY(attn_gate(a, mixed, b.ld_o, first, rows, s));
  return gemm_rows(mixed, at<T>(b.w_o), y, n, m.width, static_cast<int64_t>(b.heads) * b.vdim, b.ld_o, b.ld_o, m.width, s);
}

template <typename T>
int HybridDecoder<T>::mixer_lightning(const Branch& b, const BranchBuffers& bb, int64_t n, int64_t pos, float* y, int64_t ldp,
                                      cudaStream_t s) {
  if (chunked_lightning(b) && n >= kChunkedRows) {
    LightningArgs a;
    a.q = proj + b.col_q;
    a.k = proj + b.col_k;
    a.v = proj + b.col_v;
    a.ldp = ldp;
    a.powers = bb.powers;
    a.state = bb.state;
    a.chunk_state = chunk_state;
    a.out = o32;
    a.qb = qb;
    a.kb = kb;
    a.vb = vb;
    a.H = b.heads;
    a.dim = b.dim;
    a.vdim = b.vdim;
    a.rows = n;
    a.resume = pos > 0;
    DTRY(lightning_chunked(a, s));
  } else {
    ScanArgs a;
    a.q = proj + b.col_q;
    a.k = proj + b.col_k;
    a.v = proj + b.col_v;
    a.ldq = a.ldk = a.ldv = ldp;
    a.decay = bb.decay;
    a.silu = 1;
    a.state = bb.state;
    a.out = o32;
    a.H = a.G = b.heads;
    a.dim = b.dim;
    a.vdim = b.vdim;
    a.rows = n;
    a.resume = pos > 0;
    DTRY(recurrent_scan(a, Recurrence::kLightning, s));
  }
  const int cols = b.heads * b.vdim;
  DTRY(gated_norm_rows(o32, vec(b.w_norm), proj + b.col_g, ldp, mixed, b.ld_o, n, cols, m.eps, s));
  return gemm_rows(mixed, at<T>(b.w_o), y, n, m.width, cols, b.ld_o, b.ld_o, m.width, s);
}

template <typename T>
int HybridDecoder<T>::mixer_delta(const Branch& b, const BranchBuffers& bb, int64_t n, int64_t pos, float* y, int64_t ldp,
                                  cudaStream_t s) {
  const int64_t ldz = pad8(static_cast<int64_t>(b.heads) * b.dim), ldg = pad8(static_cast<int64_t>(b.heads) * b.vdim);
  DTRY(cast_columns(proj + b.col_a1, ldp, low_a, b.ld_a2, n, b.rank_a, s));
  DTRY(cast_columns(proj + b.col_g1, ldp, low_g, b.ld_g2, n, b.rank_g, s));
  DTRY(gemm_rows(low_a, at<T>(b.w_a2), dz, n, static_cast<int64_t>(b.heads) * b.dim, b.rank_a, b.ld_a2, b.ld_a2, ldz, s));
  DTRY(gemm_rows(low_g, at<T>(b.w_g2), dgate, n, static_cast<int64_t>(b.heads) * b.vdim, b.rank_g, b.ld_g2, b.ld_g2, ldg, s));
  DeltaPrepArgs p;
  p.proj = proj;
  p.ldp = ldp;
  p.col_q = b.col_q;
  p.col_k = b.col_k;
  p.col_v = b.col_v;
  p.col_b = b.col_b;
  p.conv_q = vec(b.conv_q);
  p.conv_k = vec(b.conv_k);
  p.conv_v = vec(b.conv_v);
  p.a_log = vec(b.a_log);
  p.dt_bias = vec(b.dt_bias);
  p.z = dz;
  p.ldz = ldz;
  p.ring = bb.ring;
  p.q = dq;
  p.k = dk;
  p.v = dv;
  p.logg = dlog;
  p.beta = dbeta;
  p.H = b.heads;
  p.G = b.kv_heads;
  p.dim = b.dim;
  p.vdim = b.vdim;
  p.taps = b.taps;
  p.rows = n;
  p.pos = pos;
  DTRY(delta_prep(p, s));
  DTRY(delta_ring_store(p, s));
  if (delta_chunked_ok(b.dim, b.vdim) && n >= kChunkedRows) {
    DeltaChunkArgs a;
    a.q = dq;
    a.k = dk;
    a.v = dv;
    a.logg = dlog;
    a.beta = dbeta;
    a.state = bb.state;
    a.out = o32;
    a.w = cw;
    a.kh = ckh;
    a.qt = cqt;
    a.u = cu;
    a.us = cus;
    a.split = m.dtype == CTDK_DTYPE_BF16 ? 1 : 0;
    a.scores = cscores;
    a.decay = cdecay;
    a.chunk_state = chunk_state;
    a.H = b.heads;
    a.G = b.kv_heads;
    a.dim = b.dim;
    a.vdim = b.vdim;
    a.rows = n;
    a.resume = pos > 0;
    DTRY(delta_chunked(a, s));
  } else {
    ScanArgs a;
    a.q = dq;
    a.k = dk;
    a.v = dv;
    a.ldq = a.ldk = static_cast<int64_t>(b.kv_heads) * b.dim;
    a.ldv = static_cast<int64_t>(b.heads) * b.vdim;
    a.logg = dlog;
    a.beta = dbeta;
    a.state = bb.state;
    a.out = o32;
    a.H = b.heads;
    a.G = b.kv_heads;
    a.dim = b.dim;
    a.vdim = b.vdim;
    a.rows = n;
    a.resume = pos > 0;
    DTRY(recurrent_scan(a, Recurrence::kDelta, s));
  }
  DTRY(gated_head_norm_rows(o32, vec(b.w_norm), dgate, ldg, mixed, b.ld_o, n, b.heads, b.vdim, m.eps, s));
  return gemm_rows(mixed, at<T>(b.w_o), y, n, m.width, static_cast<int64_t>(b.heads) * b.vdim, b.ld_o, b.ld_o, m.width, s);
}

// n <= max_portion rows at positions pos ..; `done` rows of the caller's portion came before.
template <typename T>
int HybridDecoder<T>::run_rows(const int64_t* ids, int64_t n, int64_t pos, int64_t done, const int32_t* want, int64_t n_want,
                               float* want_logits, bool last, cudaStream_t s) {
  if (m.arrangement == Arrangement::kParallel) return run_parallel_rows(ids, n, pos, done, want, n_want, want_logits, last, s);
  NormArgs<T> na;   // the pending norm: what the next norm_rows adds to the residual
  na.width = m.width;
  na.eps = m.eps;
  na.ids = ids;
  na.embed = at<T>(m.embed);
  na.ld_embed = m.ldw;
  na.w_embed = vec(m.embed_norm);
  na.h = h;
  na.ld_h = m.ldw;
  auto sandwich = [&](const float* w_pre) {
    na.x = x;
    na.x_out = x;
    na.w_pre = w_pre;
    return norm_rows(na, n, s);
  };
  auto pending = [&](const float* w_post, const float* w_y, const float* second, const float* w_y2) {
    na.ids = nullptr;
    na.y = y1;
    na.y2 = second;
    na.w_y = w_y;
    na.w_y2 = w_y2;
    na.w_post = w_post;
  };
  for (size_t l = 0; l < m.layers.size(); ++l) {
    const Layer& L = m.layers[l];
    DTRY(sandwich(vec(L.norm1)));
    if (layers_out != nullptr && l > 0 &&
        cudaMemcpyAsync(layers_out + (l - 1) * n * m.width, x, n * m.width * 4, cudaMemcpyDeviceToDevice, s) != cudaSuccess)
      return fail(CTDK_ELAUNCH, "hybrid decoder: copying the residual failed");
    DTRY(gemm_rows(h, at<T>(L.w_in), proj, n, L.n_in, m.width, m.ldw, m.ldw, L.n_in, s));
    for (size_t b = 0; b < L.branches.size(); ++b) {
      const Branch& br = L.branches[b];
      float* y = b == 0 ? y1 : y2;
      if (br.kind == BranchKind::kAttention) DTRY(mixer_attention(br, bufs[l][b], n, pos, y, L.n_in, s));
      else if (br.kind == BranchKind::kLightning) DTRY(mixer_lightning(br, bufs[l][b], n, pos, y, L.n_in, s));
      else DTRY(mixer_delta(br, bufs[l][b], n, pos, y, L.n_in, s));
    }
    if (L.branches.size() == 2) pending(vec(L.norm1b), vec(L.branches[0].w_out), y2, vec(L.branches[1].w_out));
    else pending(vec(L.norm1b), nullptr, nullptr, nullptr);
    if (L.ff > 0) {
      DTRY(sandwich(vec(L.norm2)));
      DTRY(gemm_rows(h, at<T>(L.w_gu), gu, n, 2 * L.ffp, m.width, m.ldw, m.ldw, 2 * L.ffp, s));
      DTRY(clamped_glu_rows(gu, act, n, L.ffp, L.limit, s));
      DTRY(gemm_rows(act, at<T>(L.w_down), y1, n, m.width, L.ff, L.ffp, L.ld_down, m.width, s));
      pending(vec(L.norm2b), nullptr, nullptr, nullptr);
    }
  }
  if (layers_out != nullptr) {   // the last layer's residual, which is otherwise only formed for the wanted rows
    NormArgs<T> ra = na;
    ra.x = x;
    ra.x_out = layers_out + static_cast<int64_t>(m.layers.size() - 1) * n * m.width;
    ra.w_pre = vec(m.final_norm);
    DTRY(norm_rows(ra, n, s));
  }
  return run_head(n, done, want, n_want, want_logits, last, [&](const int32_t* gather, int64_t k) {
    NormArgs<T> fa = na;
    fa.x = x;
    fa.gather = gather;
    fa.x_out = nullptr;
    fa.w_pre = vec(m.final_norm);
    return norm_rows(fa, k, s);
  }, s);
}

// The head for the wanted rows among n (see run_rows): `norm` forms h of the gathered rows.
template <typename T>
int HybridDecoder<T>::run_head(int64_t n, int64_t done, const int32_t* want, int64_t n_want, float* want_logits, bool last,
                               const std::function<int(const int32_t*, int64_t)>& norm, cudaStream_t s) {
  std::vector<int32_t> rows;
  std::vector<int64_t> dst;
  if (n_want < 0) {
    if (last) {
      rows.push_back(static_cast<int32_t>(n - 1));
      dst.push_back(-1);
    }
  } else {
    for (int64_t i = 0; i < n_want; ++i)
      if (want[i] >= done && want[i] < done + n) {
        rows.push_back(static_cast<int32_t>(want[i] - done));
        dst.push_back(i);
      }
  }
  for (size_t i0 = 0; i0 < rows.size();) {   // runs that land on consecutive output rows
    size_t i1 = i0 + 1;
    while (i1 < rows.size() && dst[i1] == dst[i1 - 1] + 1 && static_cast<int64_t>(i1 - i0) < max_portion) ++i1;
    const int64_t k = static_cast<int64_t>(i1 - i0);
    if (cudaMemcpyAsync(want_dev, rows.data() + i0, k * 4, cudaMemcpyHostToDevice, s) != cudaSuccess)
      return fail(CTDK_ELAUNCH, "hybrid decoder: copying the wanted rows failed");
    DTRY(norm(want_dev, k));
    DTRY(gemm_rows(h, at<T>(m.head), dst[i0] < 0 ? logits : want_logits + dst[i0] * vocab, k, vocab, m.width, m.ldw, m.ldw, vocab, s));
    i0 = i1;
  }
  return CTDK_OK;
}

template <typename T>
int HybridDecoder<T>::portion(const int64_t* ids, int64_t n, int64_t pos, const int32_t* want, int64_t n_want, float* want_logits,
                              cudaStream_t s) {
  CTDK_REQUIRE(layers_out == nullptr || n <= max_portion, "hybrid decoder: a traced portion must fit into max_portion");
  for (int64_t done = 0; done < n; done += max_portion) {
    const int64_t k = std::min(max_portion, n - done);
    DTRY(run_rows(ids + done, k, pos + done, done, want, n_want, want_logits, done + k == n, s));
  }
  return CTDK_OK;
}

template <typename T>
TokenArgs HybridDecoder<T>::token_args() const {
  TokenArgs a{};
  a.phases = phases_dev;
  a.n_phases = static_cast<int>(phases.size());
  a.width = m.width;
  a.eps = m.eps;
  a.embed = at<T>(m.embed);
  a.ld_embed = m.ldw;
  a.w_embed = m.arrangement == Arrangement::kSandwich ? vec(m.embed_norm) : nullptr;
  a.embed_scale = m.embed_scale;
  a.vocab = vocab;
  a.cur_token = cur_token;
  a.counters = counters;
  a.sync = sync;
  a.sync_words = static_cast<int>(sync_words);
  a.n_tokens = 1;
  a.status = device_status_word();
  return a;
}

template <typename T>
int HybridDecoder<T>::token_forward(cudaStream_t s) {
  const TokenArgs a = token_args();
  CTDK_REQUIRE(a.status != nullptr, "hybrid decoder: no status word");
  return launch_token_kernel<T>(a, m.arrangement == Arrangement::kParallel, token_ctas, token_smem, s);
}

template <typename T>
int HybridDecoder<T>::burst(int64_t n, int64_t* out_tokens, cudaStream_t s) {
  TokenArgs a = token_args();
  CTDK_REQUIRE(a.status != nullptr && n < (1 << 20), "hybrid decoder: too many tokens in one burst");
  a.out_tokens = out_tokens;
  a.out_offset = static_cast<int>(generated);
  a.n_tokens = static_cast<int>(n);
  return launch_token_kernel<T>(a, m.arrangement == Arrangement::kParallel, token_ctas, token_smem, s);
}

namespace {

int check_sizes(const Model* m, int64_t max_seq, int64_t max_portion) {
  CTDK_REQUIRE(m != nullptr && max_seq > 0 && max_seq < (1 << 24) && max_portion > 0, "hybrid decoder: bad arguments");
  return CTDK_OK;
}

template <typename T>
int64_t workspace_bytes(const Model& m, int64_t max_seq, int64_t max_portion) {
  HybridDecoder<T> d;
  d.m = m;
  d.vocab = m.vocab;
  d.max_seq = static_cast<int>(max_seq);
  d.max_portion = std::min(max_portion, max_seq);
  Bump b(nullptr);
  return d.carve(b) == CTDK_OK ? b.used : -1;
}

template <typename T>
int create(const Model& m, const void* params, void* workspace, int64_t bytes, int64_t max_seq, int64_t max_portion, void** out) {
  HybridDecoder<T>* d = new (std::nothrow) HybridDecoder<T>();
  if (d == nullptr) return fail(CTDK_ENOMEM, "hybrid decoder: out of host memory");
  d->m = m;
  d->vocab = m.vocab;
  d->max_seq = static_cast<int>(max_seq);
  d->max_portion = std::min(max_portion, max_seq);
  d->params = static_cast<const char*>(params);
  Bump b(workspace);
  int rc = d->carve(b);
  if (rc == CTDK_OK && b.used > bytes) rc = fail(CTDK_EINVAL, "hybrid decoder: workspace too small");
  if (rc == CTDK_OK) rc = d->build_phases();
  // stale rows of the packed attention buffer must be finite, everything else is written before it is read
  if (rc == CTDK_OK && cudaMemsetAsync(workspace, 0, b.used, cudaStreamPerThread) != cudaSuccess)
    rc = fail(CTDK_ELAUNCH, "hybrid decoder: clearing the workspace failed");
  if (rc == CTDK_OK) rc = d->upload(cudaStreamPerThread);
  if (rc != CTDK_OK) {
    delete d;
    return rc;
  }
  *out = static_cast<DecoderBase*>(d);
  return CTDK_OK;
}

}  // namespace
}  // namespace hybrid
}  // namespace ctdk

using namespace ctdk;
using namespace ctdk::hybrid;

extern "C" {

int64_t ctdk_hybrid_workspace_bytes(void* model, int64_t max_seq, int64_t max_portion) {
  const Model* m = static_cast<const Model*>(model);
  if (check_sizes(m, max_seq, max_portion) != CTDK_OK) return -1;
  return m->dtype == CTDK_DTYPE_BF16 ? workspace_bytes<__nv_bfloat16>(*m, max_seq, max_portion)
                                     : workspace_bytes<float>(*m, max_seq, max_portion);
}

int ctdk_hybrid_decode_create(void* model, const void* params, void* workspace, int64_t bytes, int64_t max_seq, int64_t max_portion,
                              void** decoder) {
  CTDK_REQUIRE(model && params && workspace && decoder, "ctdk_hybrid_decode_create: null pointer");
  CTDK_REQUIRE((reinterpret_cast<uintptr_t>(params) & 255u) == 0 && (reinterpret_cast<uintptr_t>(workspace) & 255u) == 0,
               "ctdk_hybrid_decode_create: arenas must be 256-byte aligned");
  const Model* m = static_cast<const Model*>(model);
  const int rc = check_sizes(m, max_seq, max_portion);
  if (rc != CTDK_OK) return rc;
  return m->dtype == CTDK_DTYPE_BF16 ? create<__nv_bfloat16>(*m, params, workspace, bytes, max_seq, max_portion, decoder)
                                     : create<float>(*m, params, workspace, bytes, max_seq, max_portion, decoder);
}

int ctdk_hybrid_trace_layers(void* decoder, float* out) {
  CTDK_REQUIRE(decoder != nullptr, "ctdk_hybrid_trace_layers: null decoder");
  DecoderBase* base = static_cast<DecoderBase*>(decoder);
  if (auto* d = dynamic_cast<HybridDecoder<__nv_bfloat16>*>(base)) d->layers_out = out;
  else if (auto* f = dynamic_cast<HybridDecoder<float>*>(base)) f->layers_out = out;
  else return fail(CTDK_EINVAL, "ctdk_hybrid_trace_layers: not a layer-list decoder");
  return CTDK_OK;
}

}  // extern "C"
