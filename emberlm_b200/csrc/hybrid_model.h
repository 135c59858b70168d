// Description of a layer-list decoder (the "hybrid" family): what config.json says, and where every
// tensor lies in the parameter arena. Host side only.
#pragma once

#include <cstdint>
#include <string>
#include <vector>

#include "../../include/ctdk.h"

namespace ctdk {
namespace hybrid {

// Rotary positions on the first `dims` dimensions of a head, interleaved pairs (2i, 2i + 1), with
// optional wavelength-dependent frequency scaling.
struct RopeSpec {
  int dims = 0;
  double base = 10000.0;
  bool scaled = false;
  double factor = 1.0, low = 1.0, high = 1.0, original = 1.0;
  double frequency(int i) const;   // of pair i, scaled
  bool operator==(const RopeSpec& o) const {
    return dims == o.dims && base == o.base && scaled == o.scaled &&
           (!scaled || (factor == o.factor && low == o.low && high == o.high && original == o.original));
  }
};

enum class BranchKind { kAttention, kLightning, kChannelDelta, kLatent, kWkv };

// One token mixer reading the layer's normed input. Offsets are bytes into the arena, columns are
// positions inside the layer's stacked input projection. Fields a kind does not have stay 0.
struct Branch {
  BranchKind kind;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int col_q = 0, col_k = 0, col_v = 0, col_g = 0;   // attention: q, k, gate per head; lightning: q, k, v, gate
  int64_t w_o = 0;                                  // [width, heads * vdim]
  int64_t ld_o = 0;
  int64_t w_out = -1;                               // norm of the branch's output when two branches are averaged
  // attention: values are the unrotated keys, sigmoid gate per head
  float scale = 1.0f;
  int chunk = 0;                                    // 0: all earlier positions
  RopeSpec rope;
  int64_t b_q = 0, b_k = 0;
  // lightning: per-head constant decay, one norm over all heads, elementwise sigmoid gate
  std::vector<float> decay;
  int64_t w_norm = 0;                               // lightning [heads * vdim]; channel delta [vdim]
  // channel delta: short convolutions, low-rank decay and gate
  int taps = 0, col_b = 0, col_a1 = 0, col_g1 = 0, rank_a = 0, rank_g = 0;
  int64_t conv_q = 0, conv_k = 0, conv_v = 0, a_log = 0, dt_bias = 0, w_a2 = 0, ld_a2 = 0, w_g2 = 0, ld_g2 = 0;
  // latent attention: col_q and col_k are the down projections of queries and keys (the latter kv_rank
  // columns of latent, then the shared rotated key part), col_g one gate per head
  int rot_dim = 0, kv_rank = 0, q_rank = 0;
  int64_t q_norm = 0, kv_norm = 0;                  // [q_rank], [kv_rank]
  int64_t w_uq = 0, ld_uq = 0;                      // [heads * (dim + rot_dim), q_rank]
  int64_t w_ukv = 0, ld_ukv = 0;                    // unrotated key rows, from row_uv on value rows; kv_rank columns
  int row_uv = 0, n_ukv = 0;
  // time mixing with a bonus (wkv): r, k, v, gate, low-rank decay rows of the stack, each with its own mix;
  // w_norm is [heads * dim]
  static constexpr int kMixes = 5;
  int col_mix[kMixes] = {0, 0, 0, 0, 0};            // r, k, v, g, w1
  int64_t mu[kMixes] = {0, 0, 0, 0, 0};
  int64_t w_w2 = 0, ld_w2 = 0, w0 = 0, bonus = 0;
  int rank_w = 0;
};

// Mixture of experts: `experts` GLUs, then `identity` outputs that return their input. Expert e's gate rows,
// then its up rows (effp each) are rows e * 2 * effp .. of w_gu; its down rows start at e * pad8(width).
struct Moe {
  int experts = 0, identity = 0, top = 0, groups = 1, keep = 1;
  int eff = 0, effp = 0;
  int64_t w_gu = 0, w_down = 0, ld_down = 0, correction = 0;
  int sff = 0, sffp = 0;                            // shared expert (0: none)
  int64_t w_sdown = 0, ld_sdown = 0;
  int outputs() const { return experts + identity; }
};

// How a layer's sublayers sit around the residual: one after the other between norms, or both from one norm.
enum class Arrangement { kSandwich, kParallel };
enum class FeedForward { kNone, kClampedGlu, kGeluGlu, kMoe };

struct Layer {
  int64_t norm1 = 0, norm1b = 0, norm2 = 0, norm2b = 0;
  int64_t w_in = 0;        // stacked input projection of all branches [n_in, ld(width)]
  int n_in = 0;
  std::vector<Branch> branches;
  int ff = 0, ffp = 0;     // feed-forward width (0: none) and its padded column count
  float limit = 0.0f;
  int64_t w_gu = 0, w_down = 0, ld_down = 0;   // gate rows then up rows [2 * ffp, ld(width)]; [width, ld(ff)]
  FeedForward ffn = FeedForward::kNone;
  // parallel arrangement: token shift in front of the mixer; what reads the unshifted norm is one stack
  // (sublayer gates, gate / up rows of a dense or shared feed-forward, router)
  int64_t shift = 0, b_rg1 = 0, b_rg2 = 0;
  int64_t w_side = 0;
  int n_side = 0, col_rg1 = 0, col_rg2 = 0, col_gu = 0, col_router = 0, col_sg = 0;
  Moe moe;
};

struct Model {
  int dtype = CTDK_DTYPE_BF16;
  int vocab = 0, width = 0;
  int64_t ldw = 0;         // row pitch of matrices with `width` columns
  float eps = 0.0f;
  Arrangement arrangement = Arrangement::kSandwich;
  int norm_groups = 1;
  float embed_scale = 1.0f;
  int64_t embed = 0, embed_norm = 0, final_norm = 0, head = 0;
  std::vector<Layer> layers;
  std::vector<ctdk_tensor_info> tensors;
  int64_t arena_bytes = 0;
  int elem() const { return dtype == CTDK_DTYPE_BF16 ? 2 : 4; }
};

inline int pad8(int64_t n) { return static_cast<int>((n + 7) / 8 * 8); }

// Throws std::runtime_error on anything it does not know.
void parse_model(const std::string& config_json, const std::string& tensors_json, int dtype, Model* out);

}  // namespace hybrid
}  // namespace ctdk
