// Choice of experts by one warp: soft-max scores, groups of neighbouring experts, renormalised weights.
#pragma once
#include "utils.cuh"

namespace {

// the largest of v[0 .. n) and its index (the lowest among equals); n <= idx when there is no number above `floor`
__device__ __forceinline__ void warp_argmax(const float* v, int n, float floor, int lane, float& best, int& bi) {
  best = floor;
  bi = 0x7fffffff;
  for (int e = lane; e < n; e += 32)
    if (v[e] > best) { best = v[e]; bi = e; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
  }
}

// sc [E] (shared memory): router logits, overwritten.  gs [groups]: room for the groups' scores.  The E experts form
// `groups` equal groups of neighbours; only experts of the `keep` groups with the largest best score can be chosen.
// weights[r] = scale * s_r / (sum of the chosen scores + 1e-20), experts in descending score.
__device__ __forceinline__ void softmax_grouped_topk(float* sc, float* gs, int E, int groups, int keep, int k, float scale,
                                                     float* weights, int64_t* idx, int lane) {
  float mx = -INFINITY;
  for (int e = lane; e < E; e += 32) mx = fmaxf(mx, sc[e]);
  mx = warp_max(mx);
  float sum = 0.f;
  for (int e = lane; e < E; e += 32) {
    const float p = expf(sc[e] - mx);
    sc[e] = p;
    sum += p;
  }
  sum = warp_sum(sum);
  __syncwarp();
  for (int e = lane; e < E; e += 32) sc[e] /= sum;
  __syncwarp();
  if (keep < groups) {
    const int per = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float b = -1.f;
      for (int i = 0; i < per; ++i) b = fmaxf(b, sc[g * per + i]);
      gs[g] = b;
    }
    __syncwarp();
    for (int r = 0; r < keep; ++r) {
      float best;
      int bi;
      warp_argmax(gs, groups, -1.f, lane, best, bi);
      __syncwarp();
      if (lane == 0 && bi < groups) gs[bi] = -2.f;         // chosen
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (gs[e / per] > -2.f) sc[e] = -1.f;
    __syncwarp();
  }
  float total = 0.f;
  for (int r = 0; r < k; ++r) {
    float best;
    int bi;
    warp_argmax(sc, E, -1.f, lane, best, bi);
    if (bi >= E) { bi = 0; best = 0.f; }                   // scores that are not numbers
    total += best;
    if (lane == 0) {
      weights[r] = best;
      idx[r] = bi;
      sc[bi] = -2.f;
    }
    __syncwarp();
  }
  const float f = scale / (total + 1e-20f);
  if (lane == 0)
    for (int r = 0; r < k; ++r) weights[r] *= f;
}

}  // namespace
