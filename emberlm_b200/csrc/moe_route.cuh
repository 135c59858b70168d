// Choice of the experts of one token by one warp, shared by the prompt and the token kernels.
#pragma once

#include <cfloat>

#include "common.cuh"

namespace ctdk {
namespace hybrid {

inline __host__ __device__ int route_scratch(int outputs, int groups) { return outputs + 2 * groups; }   // floats

// Floats as unsigned integers of the same order.
__device__ __forceinline__ uint32_t ordered(float v) {
  const uint32_t u = __float_as_uint(v);
  return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}

// z: `outputs` router logits; scratch: memory of this warp alone. Scores are softmax(z). The choice goes by
// score + correction, restricted to the `keep` groups (of outputs / groups neighbours each) whose best
// choice score is largest; the lower index wins a tie. Writes the `top` chosen outputs in order of choice
// and score / (sum of the chosen scores + 1e-20). K: outputs per lane that are held in registers
// (outputs <= 32 K).
template <int K>
__device__ __forceinline__ void route_outputs(const float* z, const float* correction, int outputs, int groups, int keep, int top,
                                              float* scratch, int32_t* index, float* weight) {
  const int lane = threadIdx.x & 31, per = outputs / groups;
  float *shared_choice = scratch, *best = scratch + outputs, *kept = best + groups;
  float e[K], choice[K];
  float m = -FLT_MAX;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int i = lane + 32 * k;
    e[k] = i < outputs ? z[i] : -FLT_MAX;
    choice[k] = i < outputs ? correction[i] : 0.0f;
    m = fmaxf(m, e[k]);
  }
  m = warp_max(m);
  float l = 0.0f;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    e[k] = lane + 32 * k < outputs ? expf(e[k] - m) : 0.0f;
    l += e[k];
  }
  const float inv = 1.0f / warp_sum(l);
#pragma unroll
  for (int k = 0; k < K; ++k) choice[k] = lane + 32 * k < outputs ? fmaf(e[k], inv, choice[k]) : -INFINITY;
  if (keep < groups) {
#pragma unroll
    for (int k = 0; k < K; ++k)
      if (lane + 32 * k < outputs) shared_choice[lane + 32 * k] = choice[k];
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      float b = -FLT_MAX;
#pragma unroll 4
      for (int k = 0; k < per; ++k) b = fmaxf(b, shared_choice[g * per + k]);
      best[g] = b;
    }
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      const float mine = best[g];
      int ahead = 0;
#pragma unroll 4
      for (int k = 0; k < groups; ++k) ahead += (best[k] > mine || (best[k] == mine && k < g)) ? 1 : 0;
      kept[g] = ahead < keep ? 1.0f : 0.0f;
    }
    __syncwarp();
#pragma unroll
    for (int k = 0; k < K; ++k) {
      const int i = lane + 32 * k;
      if (i < outputs && kept[i / per] == 0.0f) choice[k] = -INFINITY;
    }
  }
  float sum = 0.0f, mine = 0.0f;   // mine: the score of choice number `lane`
  int chosen = 0;
  for (int c = 0; c < top; ++c) {
    float v = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int k = 0; k < K; ++k)
      if (choice[k] > v) {
        v = choice[k];
        at = lane + 32 * k;
      }
    const uint32_t key = ordered(v), most = __reduce_max_sync(0xffffffffu, key);
    at = static_cast<int>(__reduce_min_sync(0xffffffffu, key == most ? static_cast<uint32_t>(at) : 0x7fffffffu));
    if (at >= outputs) at = 0;   // only when the logits are not numbers
    float score = 0.0f;
#pragma unroll
    for (int k = 0; k < K; ++k)
      if (at == lane + 32 * k) {
        score = e[k];
        choice[k] = -INFINITY;
      }
    score = __shfl_sync(0xffffffffu, score, at & 31) * inv;
    sum += score;
    if (lane == c) {
      mine = score;
      chosen = at;
    }
  }
  if (lane < top) {
    index[lane] = chosen;
    weight[lane] = mine / (sum + 1e-20f);
  }
  __syncwarp();
}
// Rare: kept out of its callers' registers.
__device__ __noinline__ inline void route_many(const float* z, const float* correction, int outputs, int groups, int keep, int top,
                                               float* scratch, int32_t* index, float* weight) {
  route_outputs<32>(z, correction, outputs, groups, keep, top, scratch, index, weight);
}
__device__ __forceinline__ void route_token(const float* z, const float* correction, int outputs, int groups, int keep, int top,
                                            float* scratch, int32_t* index, float* weight) {
  if (outputs <= 64) route_outputs<2>(z, correction, outputs, groups, keep, top, scratch, index, weight);
  else if (outputs <= 256) route_outputs<8>(z, correction, outputs, groups, keep, top, scratch, index, weight);
  else route_many(z, correction, outputs, groups, keep, top, scratch, index, weight);
}

}  // namespace hybrid
}  // namespace ctdk
