// One-token pass of the layer-list family: a list of phases that one persistent cooperative kernel
// walks, separated by grid barriers (hybrid_token.cu). The list is built once per decoder.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace ctdk {
namespace hybrid {

constexpr int kAttnSplits = 16;   // most key ranges per key/value head
constexpr int kAttnStats = 2;     // running maximum and sum in front of a partial output

enum StageKind { kStageNorm = 0, kStageGlu = 1, kStageMixed = 2 };
enum TokenBranchKind { kTokAttention = 0, kTokLightning = 1, kTokDelta = 2 };

// One rows-times-vector product: y[n] = W[n, 0..K) . staged[in ..]
struct TokenGemv {
  const void* W;
  float* y;
  int rows, K, in;   // K is the padded row pitch (padding of W and of the staged vector is zero)
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
};

struct TokenPhase {
  int is_mix;
  // products
  int stage, n_gemv, wpr, is_head;
  TokenGemv gemv[2];
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
  const float* w_embed;
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
int token_grid(size_t smem, int* grid);   // CTAs of the cooperative launch
template <typename T>
int launch_token_kernel(const TokenArgs& a, int grid, size_t smem, cudaStream_t s);

}  // namespace hybrid
}  // namespace ctdk
