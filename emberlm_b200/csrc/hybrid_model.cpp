// Reader of the layer-list model description (hybrid_model.h): config.json plus the tensor shapes.
#include <cmath>
#include <cstring>
#include <new>
#include <stdexcept>

#include "../../include/ctdk_util/minijson.hpp"
#include "common.cuh"
#include "hybrid_model.h"

namespace ctdk {
namespace hybrid {
namespace {

using minijson::Value;

[[noreturn]] void bad(const std::string& what) { throw std::runtime_error("hybrid model: " + what); }

int positive(const Value& v, const char* key) {
  const double d = v.at(key).number();
  if (!(d >= 1.0 && d <= 2147483647.0) || d != std::floor(d)) bad(std::string("'") + key + "' must be a positive integer");
  return static_cast<int>(d);
}

// Hands out arena space and keeps the tensor table, checking shapes against the file's.
class Layout {
 public:
  Layout(Model* m, const Value& shapes) : m_(m), shapes_(shapes) {}

  std::vector<int64_t> shape(const std::string& name) const {
    if (!shapes_.contains(name)) bad("tensor " + name + " is missing");
    std::vector<int64_t> s;
    for (const Value& d : shapes_.at(name).at("shape").array()) s.push_back(static_cast<int64_t>(d.number()));
    return s;
  }
  int64_t vec(const std::string& name, int64_t n) { return put(name, 1, n, n, false, {n}); }
  int64_t table(const std::string& name, int64_t rows, int64_t cols) { return put(name, rows, cols, cols, false, {rows, cols}); }
  int64_t matrix(const std::string& name, int64_t rows, int64_t cols) {
    return put(name, rows, cols, pad8(cols), true, {rows, cols});
  }
  // Consecutive matrices sharing one operand: each starts on a multiple of 8 rows.
  void begin_stack(int64_t cols) {
    align();
    stack_cols_ = cols;
    stack_base_ = m_->arena_bytes;
    stack_rows_ = 0;
  }
  int stacked(const std::string& name, int64_t rows) {
    const int64_t ld = pad8(stack_cols_);
    check(name, {rows, stack_cols_});
    add(name, rows, stack_cols_, ld, stack_base_ + stack_rows_ * ld * m_->elem(), true);
    const int first = static_cast<int>(stack_rows_);
    stack_rows_ += pad8(rows);
    return first;
  }
  int end_stack(int64_t* base) {
    *base = stack_base_;
    m_->arena_bytes = stack_base_ + stack_rows_ * pad8(stack_cols_) * m_->elem();
    align();
    if (stack_rows_ > (1 << 24)) bad("a stacked projection is too large");
    return static_cast<int>(stack_rows_);
  }

 private:
  Model* m_;
  const Value& shapes_;
  int64_t stack_cols_ = 0, stack_base_ = 0, stack_rows_ = 0;

  void align() { m_->arena_bytes = (m_->arena_bytes + 255) / 256 * 256; }
  void check(const std::string& name, const std::vector<int64_t>& want) const {
    const std::vector<int64_t> have = shape(name);
    if (have != want) {
      std::string h;
      for (const int64_t d : have) h += (h.empty() ? "" : ", ") + std::to_string(d);
      bad("tensor " + name + " has shape [" + h + "], which does not fit the config");
    }
  }
  void add(const std::string& name, int64_t rows, int64_t cols, int64_t ld, int64_t offset, bool matrix) {
    ctdk_tensor_info t;
    std::memset(&t, 0, sizeof t);
    if (name.size() >= sizeof t.name) bad("tensor name too long: " + name);
    std::memcpy(t.name, name.c_str(), name.size());
    t.rows = rows;
    t.cols = cols;
    t.ld = ld;
    t.offset = offset;
    t.is_matrix = matrix ? 1 : 0;
    m_->tensors.push_back(t);
  }
  int64_t put(const std::string& name, int64_t rows, int64_t cols, int64_t ld, bool matrix, const std::vector<int64_t>& want) {
    check(name, want);
    align();
    const int64_t off = m_->arena_bytes;
    add(name, rows, cols, ld, off, matrix);
    m_->arena_bytes += rows * ld * (matrix ? m_->elem() : 4);
    align();
    return off;
  }
};

RopeSpec parse_rope(const Value& v, int dim) {
  RopeSpec r;
  r.dims = positive(v, "dims");
  r.base = v.at("base").number();
  if (r.dims % 2 != 0 || r.dims > dim) bad("rot.dims must be even and at most the head size");
  if (v.contains("scaling") && v.at("scaling").kind != Value::kNull) {
    const Value& s = v.at("scaling");
    r.scaled = true;
    r.factor = s.at("factor").number();
    r.low = s.at("low").number();
    r.high = s.at("high").number();
    r.original = s.at("original").number();
  }
  return r;
}

// null and a missing key mean the same
bool given(const Value& v, const char* key) { return v.contains(key) && v.at(key).kind != Value::kNull; }

int count_or_zero(const Value& v, const char* key) {
  return given(v, key) && v.at(key).number() != 0.0 ? positive(v, key) : 0;
}

void check_groups(const Branch& b) {
  if (b.heads % b.kv_heads != 0) bad("heads must be a multiple of kv_heads");
}

// Softmax attention inside chunks; values tied to the unrotated keys.
Branch parse_attention(const Value& v) {
  Branch b;
  b.kind = BranchKind::kAttention;
  b.heads = positive(v, "heads");
  b.kv_heads = positive(v, "kv_heads");
  check_groups(b);
  b.dim = positive(v, "dim");
  b.vdim = positive(v, "vdim");
  if (b.vdim != b.dim) bad("tied values need vdim == dim");
  if (b.dim > 1024) bad("attention head size above 1024");
  b.scale = static_cast<float>(v.at("scale").number());
  b.chunk = v.contains("mask") && v.at("mask").kind != Value::kNull ? positive(v.at("mask"), "size") : 0;
  b.rope = parse_rope(v.at("rot"), b.dim);
  return b;
}

Branch parse_lightning(const Value& v) {
  Branch b;
  b.kind = BranchKind::kLightning;
  b.heads = b.kv_heads = positive(v, "heads");
  b.dim = positive(v, "dim");
  b.vdim = positive(v, "vdim");
  for (const Value& d : v.at("decay").array()) b.decay.push_back(static_cast<float>(d.number()));
  if (static_cast<int>(b.decay.size()) != b.heads) bad("'decay' must have one value per head");
  if (b.dim > 256) bad("recurrent key size above 256");
  return b;
}

Branch parse_channel_delta(const Value& v) {
  Branch b;
  b.kind = BranchKind::kChannelDelta;
  b.heads = positive(v, "heads");
  b.kv_heads = positive(v, "kv_heads");
  check_groups(b);
  b.dim = positive(v, "dim");
  b.vdim = positive(v, "vdim");
  b.taps = positive(v, "conv");
  if (b.dim > 256) bad("recurrent key size above 256");
  return b;
}

// Keys and values read out of one latent per position; the rotated part is rotate-half over rot_dim.
Branch parse_latent(const Value& v) {
  Branch b;
  b.kind = BranchKind::kLatent;
  b.heads = b.kv_heads = positive(v, "heads");
  b.dim = positive(v, "dim");
  b.vdim = positive(v, "vdim");
  b.rot_dim = positive(v, "rot_dim");
  b.kv_rank = positive(v, "kv_rank");
  b.q_rank = positive(v, "q_rank");
  b.scale = static_cast<float>(v.at("scale").number());
  b.rope = parse_rope(v.at("rot"), b.rot_dim);
  if (b.rope.dims != b.rot_dim) bad("latent attention rotates all of rot_dim");
  if (b.kv_rank > 1024 || b.vdim > 1024 || b.dim + b.rot_dim > 1024) bad("latent attention sizes too large");
  return b;
}

Branch parse_wkv(const Value& v) {
  Branch b;
  b.kind = BranchKind::kWkv;
  b.heads = b.kv_heads = positive(v, "heads");
  b.dim = b.vdim = positive(v, "dim");
  if (b.dim > 256) bad("recurrent key size above 256");
  return b;
}

void place_latent(Branch& b, Layout& lay, const std::string& p) {
  b.col_q = lay.stacked(p + "dq", b.q_rank);
  b.col_k = lay.stacked(p + "dkv", b.kv_rank + b.rot_dim);
  b.col_g = lay.stacked(p + "g", b.heads);
}
void place_wkv(Branch& b, Layout& lay, const std::string& p) {
  b.rank_w = static_cast<int>(lay.shape(p + "w1").at(0));
  const int64_t n = static_cast<int64_t>(b.heads) * b.dim;
  const char* names[Branch::kMixes] = {"r", "k", "v", "g", "w1"};
  for (int i = 0; i < Branch::kMixes; ++i) b.col_mix[i] = lay.stacked(p + names[i], i < 4 ? n : b.rank_w);
}
void place_attention(Branch& b, Layout& lay, const std::string& p) {
  b.col_q = lay.stacked(p + "q", b.heads * b.dim);
  b.col_k = lay.stacked(p + "k", b.kv_heads * b.dim);
  b.col_g = lay.stacked(p + "g", b.heads);
}
void place_lightning(Branch& b, Layout& lay, const std::string& p) {
  b.col_q = lay.stacked(p + "q", b.heads * b.dim);
  b.col_k = lay.stacked(p + "k", b.heads * b.dim);
  b.col_v = lay.stacked(p + "v", b.heads * b.vdim);
  b.col_g = lay.stacked(p + "g", b.heads * b.vdim);
}
void place_channel_delta(Branch& b, Layout& lay, const std::string& p) {
  b.rank_a = static_cast<int>(lay.shape(p + "a1").at(0));
  b.rank_g = static_cast<int>(lay.shape(p + "g1").at(0));
  b.col_q = lay.stacked(p + "q", b.kv_heads * b.dim);
  b.col_k = lay.stacked(p + "k", b.kv_heads * b.dim);
  b.col_v = lay.stacked(p + "v", b.heads * b.vdim);
  b.col_b = lay.stacked(p + "b", b.heads);
  b.col_a1 = lay.stacked(p + "a1", b.rank_a);
  b.col_g1 = lay.stacked(p + "g1", b.rank_g);
}
// What a branch has beside its rows of the stacked projection.
void place_rest(Branch& b, Layout& lay, const std::string& p, int width) {
  if (b.kind == BranchKind::kAttention) {
    b.b_q = lay.vec(p + "q.b", b.heads * b.dim);
    b.b_k = lay.vec(p + "k.b", b.kv_heads * b.dim);
  } else if (b.kind == BranchKind::kLightning) {
    b.w_norm = lay.vec(p + "norm", b.heads * b.vdim);
  } else if (b.kind == BranchKind::kLatent) {
    b.q_norm = lay.vec(p + "dq.norm", b.q_rank);
    b.kv_norm = lay.vec(p + "dkv.norm", b.kv_rank);
    lay.begin_stack(b.q_rank);   // alone in its stack: a product takes whole groups of eight rows
    lay.stacked(p + "uq", static_cast<int64_t>(b.heads) * (b.dim + b.rot_dim));
    lay.end_stack(&b.w_uq);
    b.ld_uq = pad8(b.q_rank);
    lay.begin_stack(b.kv_rank);
    lay.stacked(p + "uk", static_cast<int64_t>(b.heads) * b.dim);
    b.row_uv = lay.stacked(p + "uv", static_cast<int64_t>(b.heads) * b.vdim);
    b.n_ukv = lay.end_stack(&b.w_ukv);
    b.ld_ukv = pad8(b.kv_rank);
  } else if (b.kind == BranchKind::kWkv) {
    const char* names[Branch::kMixes] = {"r", "k", "v", "g", "w"};
    for (int i = 0; i < Branch::kMixes; ++i) b.mu[i] = lay.vec(p + "mu." + names[i], width);
    lay.begin_stack(b.rank_w);
    lay.stacked(p + "w2", static_cast<int64_t>(b.heads) * b.dim);
    lay.end_stack(&b.w_w2);
    b.ld_w2 = pad8(b.rank_w);
    b.w0 = lay.vec(p + "w0", static_cast<int64_t>(b.heads) * b.dim);
    b.bonus = lay.table(p + "u", b.heads, b.dim);
    b.w_norm = lay.vec(p + "norm", static_cast<int64_t>(b.heads) * b.dim);
  } else {
    b.conv_q = lay.table(p + "q.conv", b.kv_heads * b.dim, b.taps);
    b.conv_k = lay.table(p + "k.conv", b.kv_heads * b.dim, b.taps);
    b.conv_v = lay.table(p + "v.conv", b.heads * b.vdim, b.taps);
    b.a_log = lay.vec(p + "A_log", b.heads);
    b.dt_bias = lay.vec(p + "dt_bias", b.heads * b.dim);
    b.w_norm = lay.vec(p + "norm", b.vdim);
    b.w_a2 = lay.matrix(p + "a2", b.heads * b.dim, b.rank_a);
    b.ld_a2 = pad8(b.rank_a);
    b.w_g2 = lay.matrix(p + "g2", b.heads * b.vdim, b.rank_g);
    b.ld_g2 = pad8(b.rank_g);
  }
  b.w_o = lay.matrix(p + "o", width, b.heads * b.vdim);
  b.ld_o = pad8(static_cast<int64_t>(b.heads) * b.vdim);
}

}  // namespace

namespace {

Moe parse_moe(const Value& v) {
  Moe e;
  const Value& r = v.at("router");
  e.experts = positive(r, "experts");
  e.identity = count_or_zero(r, "identity");
  e.top = positive(r, "top");
  if (given(r, "groups")) {
    e.groups = positive(r.at("groups"), "count");
    e.keep = positive(r.at("groups"), "keep");
  }
  if (e.outputs() % e.groups != 0) bad("router outputs must form equal groups");
  if (e.keep > e.groups || e.top > e.outputs() / e.groups * e.keep) bad("the router keeps fewer outputs than it chooses");
  if (e.outputs() > 1024 || e.top > 32) bad("more than 1024 router outputs or 32 chosen ones");
  e.eff = positive(v.at("expert"), "ff");
  e.effp = pad8(e.eff);
  if (given(v, "shared")) {
    e.sff = positive(v.at("shared"), "ff");
    e.sffp = pad8(e.sff);
  }
  return e;
}

// One norm, token shift, mixer and feed-forward side by side, each behind its own gate.
Layer parse_parallel_layer(const Model& m, const Value& lv, Layout& lay, const std::string& p) {
  const std::string mix = p + "mix.", mlp = p + "mlp.", type = lv.at("type").string();
  const int W = m.width;
  Layer L;
  L.norm1 = lay.vec(p + "norm1", W);
  L.shift = lay.vec(p + "shift", W);
  const Value& mv = lv.at("mixer");
  if (type == "latent_attention") L.branches.push_back(parse_latent(mv));
  else if (type == "wkv") L.branches.push_back(parse_wkv(mv));
  else bad("unknown mixer type '" + type + "'");
  Branch& b = L.branches[0];
  lay.begin_stack(W);
  if (b.kind == BranchKind::kLatent) place_latent(b, lay, mix);
  else place_wkv(b, lay, mix);
  L.n_in = lay.end_stack(&L.w_in);
  place_rest(b, lay, mix, W);

  if (given(lv, "mlp")) {
    const Value& f = lv.at("mlp");
    const std::string kind = f.at("kind").string();
    if (kind == "dense") {
      L.ffn = FeedForward::kGeluGlu;
      L.ff = positive(f, "ff");
      L.ffp = pad8(L.ff);
    } else if (kind == "moe") {
      L.ffn = FeedForward::kMoe;
      L.moe = parse_moe(f);
    } else {
      bad("unknown feed-forward kind '" + kind + "'");
    }
  }
  Moe& e = L.moe;
  lay.begin_stack(W);
  L.col_rg1 = lay.stacked(p + "rg1", W);
  if (L.ffn != FeedForward::kNone) L.col_rg2 = lay.stacked(p + "rg2", W);
  if (L.ffn == FeedForward::kGeluGlu || e.sff > 0) {
    const std::string q = L.ffn == FeedForward::kGeluGlu ? mlp : mlp + "shared.";
    const int ff = L.ffn == FeedForward::kGeluGlu ? L.ff : e.sff;
    L.col_gu = lay.stacked(q + "gate", ff);
    lay.stacked(q + "up", ff);
  }
  if (L.ffn == FeedForward::kMoe) {
    L.col_router = lay.stacked(mlp + "router", e.outputs());
    if (e.sff > 0) L.col_sg = lay.stacked(mlp + "shared.sg", 1);
  }
  L.n_side = lay.end_stack(&L.w_side);
  L.b_rg1 = lay.vec(p + "rg1.b", W);
  if (L.ffn != FeedForward::kNone) L.b_rg2 = lay.vec(p + "rg2.b", W);
  if (L.ffn == FeedForward::kGeluGlu) {
    L.w_down = lay.matrix(mlp + "down", W, L.ff);
    L.ld_down = L.ffp;
  } else if (L.ffn == FeedForward::kMoe) {
    e.correction = lay.vec(mlp + "correction", e.outputs());
    lay.begin_stack(W);
    for (int i = 0; i < e.experts; ++i) {
      lay.stacked(mlp + "e" + std::to_string(i) + ".gate", e.eff);
      lay.stacked(mlp + "e" + std::to_string(i) + ".up", e.eff);
    }
    lay.end_stack(&e.w_gu);
    lay.begin_stack(e.eff);
    for (int i = 0; i < e.experts; ++i) lay.stacked(mlp + "e" + std::to_string(i) + ".down", W);
    lay.end_stack(&e.w_down);
    e.ld_down = e.effp;
    if (e.sff > 0) {
      e.w_sdown = lay.matrix(mlp + "shared.down", W, e.sff);
      e.ld_sdown = e.sffp;
    }
  }
  return L;
}

void parse_parallel_model(const Value& c, Layout& lay, Model& m) {
  m.arrangement = Arrangement::kParallel;
  m.norm_groups = positive(c.at("norm"), "groups");
  if (m.width % m.norm_groups != 0) bad("norm.groups must divide the width");
  m.embed_scale = static_cast<float>(c.at("embedding").at("scale").number());
  m.embed = lay.matrix("embed", m.vocab, m.width);
  const minijson::Array& layers = c.at("layers").array();
  std::vector<int> source;   // whose weights a layer uses; every layer has a cache and state of its own
  for (size_t i = 0; i < layers.size(); ++i) {
    const double j = given(layers[i], "weights_of") ? layers[i].at("weights_of").number() : static_cast<double>(i);
    if (!(j >= 0.0 && j < static_cast<double>(layers.size())) || j != std::floor(j)) bad("'weights_of' must name a layer");
    source.push_back(static_cast<int>(j));
  }
  m.layers.resize(layers.size());
  for (size_t i = 0; i < layers.size(); ++i)
    if (source[i] == static_cast<int>(i)) m.layers[i] = parse_parallel_layer(m, layers[i], lay, "l" + std::to_string(i) + ".");
  for (size_t i = 0; i < layers.size(); ++i) {
    if (source[source[i]] != source[i]) bad("'weights_of' must name a layer with weights of its own");
    if (source[i] != static_cast<int>(i)) m.layers[i] = m.layers[source[i]];
  }
}

}  // namespace

double RopeSpec::frequency(int i) const {
  const double f = std::pow(base, -2.0 * i / dims);
  if (!scaled) return f;
  const double wavelength = 2.0 * 3.14159265358979323846 / f;
  if (wavelength < original / high) return f;
  if (wavelength > original / low) return f / factor;
  const double s = (original / wavelength - low) / (high - low);
  return (1.0 - s) * f / factor + s * f;
}

void parse_model(const std::string& config_json, const std::string& tensors_json, int dtype, Model* out) {
  const Value c = minijson::parse(config_json);
  const Value shapes = minijson::parse(tensors_json);
  const std::string arch = c.at("architecture").string();
  if (arch != "Zutalix" && arch != "Detatar") bad("unknown architecture '" + arch + "'");
  if (dtype != CTDK_DTYPE_F32 && dtype != CTDK_DTYPE_BF16) bad("unknown dtype");
  Model& m = *out;
  m = Model();
  m.dtype = dtype;
  m.vocab = positive(c, "vocab");
  m.width = positive(c, "width");
  if (m.width > 16384) bad("width above 16384");
  m.ldw = pad8(m.width);
  m.eps = static_cast<float>(c.at("norm").at("eps").number());
  Layout lay(&m, shapes);
  if (arch == "Detatar") {
    parse_parallel_model(c, lay, m);
    m.final_norm = lay.vec("final.norm", m.width);
    m.head = lay.matrix("head", m.vocab, m.width);
    return;
  }
  m.embed = lay.matrix("embed", m.vocab, m.width);
  m.embed_norm = lay.vec("embed.norm", m.width);
  int i = 0;
  for (const Value& lv : c.at("layers").array()) {
    const std::string p = "l" + std::to_string(i++) + ".", mix = p + "mix.";
    const std::string type = lv.at("type").string();
    const Value& mv = lv.at("mixer");
    Layer L;
    L.norm1 = lay.vec(p + "norm1", m.width);
    L.norm1b = lay.vec(p + "norm1b", m.width);
    lay.begin_stack(m.width);
    if (type == "parallel") {
      L.branches.push_back(parse_attention(mv.at("left")));
      L.branches.push_back(parse_lightning(mv.at("right")));
      place_attention(L.branches[0], lay, mix + "left.");
      place_lightning(L.branches[1], lay, mix + "right.");
      L.n_in = lay.end_stack(&L.w_in);
      place_rest(L.branches[0], lay, mix + "left.", m.width);
      place_rest(L.branches[1], lay, mix + "right.", m.width);
      L.branches[0].w_out = lay.vec(mix + "left.out", m.width);
      L.branches[1].w_out = lay.vec(mix + "right.out", m.width);
    } else if (type == "channel_delta") {
      L.branches.push_back(parse_channel_delta(mv));
      place_channel_delta(L.branches[0], lay, mix);
      L.n_in = lay.end_stack(&L.w_in);
      place_rest(L.branches[0], lay, mix, m.width);
    } else {
      bad("unknown mixer type '" + type + "'");
    }
    if (lv.contains("mlp") && lv.at("mlp").kind != Value::kNull) {
      const Value& f = lv.at("mlp");
      if (f.at("kind").string() != "dense") bad("unknown feed-forward kind '" + f.at("kind").string() + "'");
      L.ffn = FeedForward::kClampedGlu;
      L.ff = positive(f, "ff");
      L.ffp = pad8(L.ff);
      L.limit = static_cast<float>(f.at("limit").number());
      L.norm2 = lay.vec(p + "norm2", m.width);
      L.norm2b = lay.vec(p + "norm2b", m.width);
      lay.begin_stack(m.width);
      lay.stacked(p + "mlp.gate", L.ff);
      lay.stacked(p + "mlp.up", L.ff);
      lay.end_stack(&L.w_gu);
      L.w_down = lay.matrix(p + "mlp.down", m.width, L.ff);
      L.ld_down = L.ffp;
    }
    m.layers.push_back(L);
  }
  m.final_norm = lay.vec("final.norm", m.width);
  m.head = lay.matrix("head", m.vocab, m.width);
}

}  // namespace hybrid
}  // namespace ctdk

using ctdk::hybrid::Model;

extern "C" {

int ctdk_hybrid_open(const char* config_json, const char* tensors_json, int dtype, void** model) {
  CTDK_REQUIRE(config_json && tensors_json && model, "ctdk_hybrid_open: null pointer");
  try {
    Model* m = new Model();
    try {
      ctdk::hybrid::parse_model(config_json, tensors_json, dtype, m);
    } catch (...) {
      delete m;
      throw;
    }
    *model = m;
    return CTDK_OK;
  } catch (const std::exception& e) {
    return ctdk::fail(CTDK_EINVAL, "%s", e.what());
  }
}

int ctdk_hybrid_close(void* model) {
  delete static_cast<Model*>(model);
  return CTDK_OK;
}

int64_t ctdk_hybrid_num_tensors(void* model) {
  return model ? static_cast<int64_t>(static_cast<Model*>(model)->tensors.size()) : -1;
}

int ctdk_hybrid_tensor(void* model, int64_t i, ctdk_tensor_info* out) {
  CTDK_REQUIRE(model && out, "ctdk_hybrid_tensor: null pointer");
  const Model& m = *static_cast<Model*>(model);
  CTDK_REQUIRE(i >= 0 && i < static_cast<int64_t>(m.tensors.size()), "ctdk_hybrid_tensor: index out of range");
  *out = m.tensors[i];
  return CTDK_OK;
}

int64_t ctdk_hybrid_arena_bytes(void* model) { return model ? static_cast<Model*>(model)->arena_bytes : -1; }
int64_t ctdk_hybrid_vocab(void* model) { return model ? static_cast<Model*>(model)->vocab : -1; }

}  // extern "C"
