// Causal convolution over a few tokens, per channel, and silu.  Inputs of earlier calls come from a ring of `taps` rows per
// slot (row = position mod taps); what lies before a sequence's first token counts as zero.
#pragma once
#include "utils.cuh"

namespace {

// silu of a 16-bit model's convolution
__device__ __forceinline__ float fast_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// Channel c of the convolution after silu, at packed token t: token j of its portion, position p of its sequence.  w: the
// channel's last tap.  A: proj (columns = channels), ldp, ring [slots, taps, channels], taps, channels.
template <typename T, typename A, typename TW>
__device__ __forceinline__ float conv_silu(const A& a, int c, int t, int j, int p, int start, int slot, const TW* w,
                                           float bias = 0.f) {
  const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)t * a.ldp + c;
  const T* ring = reinterpret_cast<const T*>(a.ring) + (int64_t)slot * a.taps * a.channels + c;
  const int pm = p % a.taps, seen = min(a.taps, p - start + 1);
  float s = bias;
  for (int b0 = 0; b0 < a.taps; b0 += 4) {
    T x[4];
    float wv[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int back = b0 + u;
      x[u] = DT<T>::from_f(0.f);
      wv[u] = 0.f;
      if (back < a.taps) {                       // (rows from before the start are read and not used: `start` comes late)
        const int r = pm - back;
        x[u] = back <= j ? proj[-(int64_t)back * a.ldp] : ring[(int64_t)(r < 0 ? r + a.taps : r) * a.channels];
        wv[u] = DT<TW>::to_f(w[-back]);
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (b0 + u < seen) s = fmaf(DT<T>::to_f(x[u]), wv[u], s);
  }
  return silu(s);
}

// Eight neighbouring channels of the convolution for four tokens: every input row is read once.  TP: taps, 0 if only
// known at run time.  first: token (of the chunk) of the first output; ws [taps][ldws]: weights of these channels; bias
// [8] or null.
template <typename T, int TP, typename A>
__device__ __forceinline__ void conv_block(const A& a, int c, int t0, int row0, int p0, int start, int slot, int n,
                                           int first, const float* ws, int ldws, float (&acc)[4][8],
                                           const float* bias = nullptr) {
  const int taps = TP > 0 ? TP : a.taps;
  const T* proj = reinterpret_cast<const T*>(a.proj) + c;
  const T* ring = reinterpret_cast<const T*>(a.ring) + (int64_t)slot * taps * a.channels + c;
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[j][e] = bias != nullptr ? bias[e] : 0.f;
  auto row = [&](int rr) {
    const int rel = first - (taps - 1) + rr, p = p0 + rel, t = t0 + rel;
    uint4 raw = make_uint4(0, 0, 0, 0);
    if (p >= start && rel < n)
      raw = *reinterpret_cast<const uint4*>(t >= row0 ? proj + (int64_t)t * a.ldp
                                                      : ring + (int64_t)(p % taps) * a.channels);
    return raw;
  };
  auto use = [&](int rr, const uint4& raw) {
    const T* e8 = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = rr - j;
      if (i >= 0 && i < taps) {
        const float4 w0 = *reinterpret_cast<const float4*>(ws + i * ldws);
        const float4 w1 = *reinterpret_cast<const float4*>(ws + i * ldws + 4);
        const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[j][e] = fmaf(DT<T>::to_f(e8[e]), w[e], acc[j][e]);
      }
    }
  };
  if constexpr (TP > 0) {
    uint4 raw[TP + 3];
#pragma unroll
    for (int rr = 0; rr < TP + 3; ++rr) raw[rr] = row(rr);
#pragma unroll
    for (int rr = 0; rr < TP + 3; ++rr) use(rr, raw[rr]);
  } else {
    for (int rr = 0; rr < taps + 3; ++rr) use(rr, row(rr));
  }
}

}  // namespace
