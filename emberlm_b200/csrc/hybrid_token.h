// One-token pass of the layer-list family: a list of phases that one persistent cooperative kernel
// walks, separated by grid barriers (hybrid_token.cu). The list is built once per decoder.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace ctdk {
namespace hybrid {

constexpr int kAttnSplits = 16;   // most key ranges per key/value head
constexpr int kAttnStats = 2;     // running maximum and sum in front of a partial output
constexpr int kAttnStats4 = 4;    // the same, with room that keeps the output 16-byte aligned

constexpr int kListThreads = 512, kListWarps = kListThreads / 32;   // of a CTA that runs kStageList phases, one per SM
constexpr int kLatentHeads = 16;   // query heads that share one pass over the latent cache (bfloat16)
constexpr int kLatentHeadsF32 = 8; // the same for fp32 models
constexpr int kLatentSplits = 96;  // most position ranges per block of heads
constexpr int kLatentKeys = 32;    // cache rows staged at once
constexpr int kLatentOutRows = 32; // value rows of an output item
constexpr int kLatentOutParts = 4; // thread groups that share the merging of the ranges

enum StageKind { kStageNorm = 0, kStageGlu = 1, kStageMixed = 2, kStageList = 3 };
enum TokenBranchKind { kTokAttention = 0, kTokLightning = 1, kTokDelta = 2, kTokWkv = 3, kTokLatentKeys = 4, kTokLatentScan = 5, kTokLatentOut = 6 };

// One rows-times-vector product: y[n] = W[n, 0..K) . staged[in ..]
//   kGemvExpertUp    rows r of chosen output r / per: row r % per of that expert's `pitch` rows (identity: skipped)
//   kGemvExpertDown  row r: the sum over the chosen experts of row r of their `pitch` rows with staged[in + slot K ..],
//                    plus W2[r, 0..K2) . staged[in2 ..] (W2 may be null), plus (identity weights) h[r]
enum GemvMode { kGemvPlain = 0, kGemvExpertUp = 1, kGemvExpertDown = 2 };
struct TokenGemv {
  const void* W;
  float* y;
  int rows, K, in;   // K is the padded row pitch (padding of W and of the staged vector is zero)
  int mode, per, pitch, top, experts, K2, in2;
  const void* W2;
  const float* h;
};

// What a kStageList phase puts into the staged vector, in order (`at`: first float; padded with zeros to `ld`).
enum StageOpKind {
  kOpShiftNorm,     // TokenShift below: h at 0, the shifted row at ldw, the mixes behind it
  kOpRmsNorm,       // n values of src, normed, * w
  kOpCopy,          // n values of src
  kOpRoute,         // src2 (width values) padded to ld; chooses the experts from the n router logits src, correction w (kept until the next choice)
  kOpGelu,          // gelu(src[c]) src[ld + c], c < n
  kOpShared,        // sigmoid(src2[0]) silu(src[c]) src[ld + c], c < n
  kOpExperts,       // per chosen expert: weight silu(gate) up, n columns from its 2 n values of src
  kOpHeadNorm,      // per head of branch 0: src normed over dim, * w * silu(src2)
  kOpLatentStore    // the position's cache row of branch 0 (one CTA)
};
struct StageOp {
  int kind, at, n, ld;
  const float *src, *src2, *w;
};
constexpr int kMaxGemv = 6, kMaxOps = 4, kTokenMixes = 5;

// Residual and norm of the parallel arrangement (see ShiftNormArgs). state: [2 slots][h, m][width], a
// position reads the slot of the one before and writes its own (slot = position mod 2).
struct TokenShift {
  int groups, wpg, n_mix, ld, red;   // red: first float of the reduction scratch
  int vec;                           // columns can be taken four at a time
  const float *x, *y1, *y2, *z1, *z2, *b1, *b2, *w, *shift, *mu[kTokenMixes];
  float *x_out, *h_out, *state;
};

// A mixer branch: what the mix phase computes and what the output projection stages from it.
struct TokenBranch {
  int kind, items;
  int H, G, dim, vdim;
  int col_q, col_k, col_v, col_g;
  float* out;            // [H * vdim]: attention gated, recurrences raw
  int stage_at;          // offset of this branch in the staged vector
  // attention
  const float *b_q, *b_k;
  const float2* table;
  int rot_pairs, chunk;
  float scale;
  void* cache;
  float* part;           // [H][kAttnSplits][dim + kAttnStats]
  unsigned int* arrive;  // [G]
  // recurrences
  const float* decay;
  float* state;
  const float* w_norm;
  // delta
  int taps, col_b, col_a1, col_g1, rank_a, rank_g;
  const float *conv_q, *conv_k, *conv_v, *a_log, *dt_bias;
  const void *w_a2, *w_g2;
  float* ring;
  float* gate;           // [H * vdim] output gate before the sigmoid
  // wkv
  int col_r, col_w1, rank_w;
  const void* w_w2;
  const float *w0, *bonus;
  // latent attention
  int rot_dim, kv_rank, rot_col, ld_cache, ld_ukv, row_uv, splits, blocks, buffers;   // buffers: cache tiles in flight (1 or 2)
  const void* w_ukv;
  const float *kv_norm, *q_up;   // queries [H][dim + rot_dim]
  void* q_abs;           // [H][ld_cache] queries against the cache rows, scaled: fp32, or two bfloat16 planes
};

struct TokenPhase {
  int is_mix;
  // products
  int stage, n_gemv, wpr, is_head;
  TokenGemv gemv[kMaxGemv];
  // kStageList phases: staging, products and the items of branch 0 in one phase
  int n_ops;
  StageOp op[kMaxOps];
  TokenShift shift;
  int route_groups, route_keep, route_top;
  const void* extra;     // weights of the items, for the prefetch
  int64_t extra_bytes;
  int first_token;       // kStageNorm: x comes from the embedding
  const float *x, *y, *y2, *w_y, *w_y2, *w_post, *w_pre;
  float* x_out;
  const float* gu;
  int ffp;
  float limit;
  // mixing
  int n_branch;
  TokenBranch br[2];
  const float* proj;
  int prefetch;          // phase whose weights this one requests into L2, or -1
};

struct TokenArgs {
  const TokenPhase* phases;
  int n_phases, width;
  float eps;
  const void* embed;
  int64_t ld_embed;
  const float* w_embed;  // norm of the embedding, or null: times embed_scale
  float embed_scale;
  int vocab;
  int64_t* cur_token;
  int* counters;
  unsigned int* sync;        // barrier words, the two arg-max words at [128], head arrivals from [256]
  int sync_words;
  int64_t* out_tokens;       // null: one token, logits only
  int out_offset, n_tokens;
  int* status;
};

constexpr int kTokenSyncWords = 256;

// Shared memory the kernel needs for a phase list (bytes), from the largest staged vector (floats).
size_t token_smem_bytes(int stage_floats, const TokenPhase* phases, int n);
template <typename T>
int token_grid(size_t smem, bool list, int* grid);   // CTAs of the cooperative launch; list: kStageList phases only
template <typename T>
int launch_token_kernel(const TokenArgs& a, bool list, int grid, size_t smem, cudaStream_t s);

}  // namespace hybrid
}  // namespace ctdk
