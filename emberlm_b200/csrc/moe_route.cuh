// Choice of the experts of one token by one warp, shared by the prompt and the token kernels.
#pragma once

#include <cfloat>

#include "common.cuh"

namespace ctdk {
namespace hybrid {

inline __host__ __device__ int route_scratch(int outputs, int groups) { return outputs + 2 * groups; }   // floats

// z: `outputs` router logits; scratch: memory of this warp alone. Scores are softmax(z). The choice goes by
// score + correction, restricted to the `keep` groups (of outputs / groups neighbours each) whose best
// choice score is largest; the lower index wins a tie. Writes the `top` chosen outputs in order of choice
// and score / (sum of the chosen scores + 1e-20).
__device__ __forceinline__ void route_token(const float* z, const float* correction, int outputs, int groups, int keep, int top,
                                            float* scratch, int32_t* index, float* weight) {
  const int lane = threadIdx.x & 31, per = outputs / groups;
  float *choice = scratch, *best = choice + outputs, *kept = best + groups;
  float m = -FLT_MAX;
  for (int i = lane; i < outputs; i += 32) m = fmaxf(m, z[i]);
  m = warp_max(m);
  float l = 0.0f;
  for (int i = lane; i < outputs; i += 32) l += expf(z[i] - m);
  const float inv = 1.0f / warp_sum(l);
  __syncwarp();
  for (int i = lane; i < outputs; i += 32) choice[i] = fmaf(expf(z[i] - m), inv, correction[i]);
  __syncwarp();
  if (keep < groups) {
    for (int g = lane; g < groups; g += 32) {
      float b = -FLT_MAX;
      for (int k = 0; k < per; ++k) b = fmaxf(b, choice[g * per + k]);
      best[g] = b;
    }
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      int ahead = 0;
      for (int k = 0; k < groups; ++k) ahead += (best[k] > best[g] || (best[k] == best[g] && k < g)) ? 1 : 0;
      kept[g] = ahead < keep ? 1.0f : 0.0f;
    }
    __syncwarp();
    for (int i = lane; i < outputs; i += 32)
      if (kept[i / per] == 0.0f) choice[i] = -INFINITY;
    __syncwarp();
  }
  float sum = 0.0f, mine = 0.0f;   // mine: the score of choice number `lane`
  for (int k = 0; k < top; ++k) {
    float v = -INFINITY;
    int at = outputs;
    for (int i = lane; i < outputs; i += 32)
      if (choice[i] > v) {
        v = choice[i];
        at = i;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, v, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ov > v || (ov == v && oa < at)) {
        v = ov;
        at = oa;
      }
    }
    if (at >= outputs) at = 0;   // only when the logits are not numbers
    const float score = expf(z[at] - m) * inv;
    sum += score;
    if (lane == k) mine = score;
    __syncwarp();
    if (lane == 0) {
      choice[at] = -INFINITY;
      index[k] = at;
    }
    __syncwarp();
  }
  if (lane < top) weight[lane] = mine / (sum + 1e-20f);
  __syncwarp();
}

}  // namespace hybrid
}  // namespace ctdk
