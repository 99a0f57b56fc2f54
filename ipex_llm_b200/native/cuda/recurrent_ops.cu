// What recurrent layers share around their recurrences, sm_100a.
//
//   ring_tail         the last inputs of short convolutions into the slot's ring
//   gated_norm        per head: o / rms(o) * w * gate, the gate silu or a sigmoid, w shared by the heads or one per column
//   gated_group_norm  y * silu(z), then an RMS norm in equal parts that need not be heads, times w
#include "common/state_cols.cuh"
#include "common/utils.cuh"

namespace {

constexpr int kThreads = 256;

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

template <typename T>
__global__ void __launch_bounds__(kThreads) ring_tail_kernel(const T* __restrict__ proj, int64_t ldp, T* ring,
                                                             const int* __restrict__ slots, const int* __restrict__ pos,
                                                             const int* __restrict__ seq_row,
                                                             const int* __restrict__ seq_len, int channels, int taps) {
  const int seq = blockIdx.y, len = seq_len[seq], row0 = seq_row[seq], n = min(len, taps);
  const int c = blockIdx.x * kThreads + threadIdx.x, slot = slots[row0], p0 = pos[row0];
  if (c >= channels) return;
  ring += (int64_t)slot * taps * channels + c;
  proj += c;
  for (int j = len - n; j < len; ++j) ring[(int64_t)((p0 + j) % taps) * channels] = proj[(int64_t)(row0 + j) * ldp];
}

// N neighbouring values
template <typename T, int N>
__device__ __forceinline__ void load_pack(const T* p, float (&v)[N]) {
  if constexpr (N == 4 && sizeof(T) == 2) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
#pragma unroll
    for (int c = 0; c < N; ++c) v[c] = DT<T>::to_f(reinterpret_cast<const T*>(&raw)[c]);
  } else {
#pragma unroll
    for (int c = 0; c < N; ++c) v[c] = DT<T>::to_f(p[c]);
  }
}
template <typename T, int N>
__device__ __forceinline__ void store_pack(T* p, const float (&v)[N]) {
  if constexpr (N == 4 && sizeof(T) == 2) {
    __align__(8) T y[N];
#pragma unroll
    for (int c = 0; c < N; ++c) y[c] = DT<T>::from_f(v[c]);
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(y);
  } else {
#pragma unroll
    for (int c = 0; c < N; ++c) p[c] = DT<T>::from_f(v[c]);
  }
}

// A warp per (token, head); VEC: four neighbouring columns per lane and step.  The result may take the place of the gates.
template <typename T, bool VEC, bool SIGMOID>
__global__ void __launch_bounds__(kThreads) gated_norm_kernel(const float* __restrict__ o, const T* gate, int64_t ldg,
                                                              const T* __restrict__ w, int w_head, T* out, int64_t ldo,
                                                              int64_t rows, int heads, int V, float eps, float scale) {
  constexpr int N = VEC ? 4 : 1;
  const int64_t r = (int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= rows) return;
  const int64_t t = r <= 0x7fffffff ? (int64_t)((uint32_t)r / (uint32_t)heads) : r / heads;
  const int h = (int)(r - t * heads);
  const float* src = o + r * V;
  const T* gt = gate + t * ldg + (int64_t)h * V;
  const T* wt = w + (int64_t)h * w_head;
  T* dst = out + t * ldo + (int64_t)h * V;
  float x[N], gv[N], wv[N], ss = 0.f;
  for (int i = lane * N; i < V; i += 32 * N) {
    load_cols<N>(src + i, x);
#pragma unroll
    for (int c = 0; c < N; ++c) ss = fmaf(x[c], x[c], ss);
  }
  const float inv = scale / sqrtf(warp_sum(ss) / (float)V + eps);
  for (int i = lane * N; i < V; i += 32 * N) {
    load_cols<N>(src + i, x);
    load_pack<T, N>(gt + i, gv);
    load_pack<T, N>(wt + i, wv);
#pragma unroll
    for (int c = 0; c < N; ++c) x[c] = x[c] * inv * wv[c] * (SIGMOID ? sigmoidf(gv[c]) : silu(gv[c]));
    store_pack<T, N>(dst + i, x);
  }
}

// CTA = one part of one token.
template <typename T, int N>
__global__ void __launch_bounds__(kThreads) gated_group_norm_kernel(const float* __restrict__ y, const T* __restrict__ z,
                                                                    int64_t ldz, const T* __restrict__ w, T* __restrict__ out,
                                                                    int64_t ldo, int width, int part, float eps) {
  __shared__ float red[kThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int c0 = blockIdx.y * part, tid = threadIdx.x, nt = blockDim.x;
  const float* yr = y + t * width + c0;
  const T* zr = z + t * ldz + c0;
  const T* wr = w + c0;
  T* dst = out + t * ldo + c0;
  constexpr int kKeep = 4;              // packs a thread keeps in registers
  float v[kKeep][N], ss = 0.f;
  auto gated = [&](int i, float (&x)[N]) {
    float g[N];
    load_cols<N>(yr + i, x);
    load_pack<T, N>(zr + i, g);
#pragma unroll
    for (int c = 0; c < N; ++c) x[c] *= silu(g[c]);
  };
#pragma unroll
  for (int k = 0; k < kKeep; ++k) {
    const int i = (tid + k * nt) * N;
    if (i < part) {
      gated(i, v[k]);
#pragma unroll
      for (int c = 0; c < N; ++c) ss = fmaf(v[k][c], v[k][c], ss);
    }
  }
  for (int i = (tid + kKeep * nt) * N; i < part; i += nt * N) {
    float x[N];
    gated(i, x);
#pragma unroll
    for (int c = 0; c < N; ++c) ss = fmaf(x[c], x[c], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = warp_sum((tid & 31) < nt / 32 ? red[tid & 31] : 0.f);
  const float inv = 1.0f / sqrtf(ss / (float)part + eps);
  auto put = [&](int i, const float (&x)[N]) {
    float wv[N], r[N];
    load_pack<T, N>(wr + i, wv);
#pragma unroll
    for (int c = 0; c < N; ++c) r[c] = x[c] * inv * wv[c];
    store_pack<T, N>(dst + i, r);
  };
#pragma unroll
  for (int k = 0; k < kKeep; ++k) {
    const int i = (tid + k * nt) * N;
    if (i < part) put(i, v[k]);
  }
  for (int i = (tid + kKeep * nt) * N; i < part; i += nt * N) {
    float x[N];
    gated(i, x);
    put(i, x);
  }
}

}  // namespace

// The last convolution inputs (columns of proj) of every sequence into its slot's ring [slots, taps, channels], after
// everything that reads the ring.
IPEX_API int ipex_ring_tail(const void* proj, int64_t ldp, void* ring, const int* slot, const int* pos, const int* seq_row,
                            const int* seq_len, int seqs, int channels, int taps, int dtype, void* stream) {
  if (seqs < 1 || seqs > 65535 || channels < 1 || taps < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ring_tail_kernel<T><<<dim3((channels + kThreads - 1) / kThreads, seqs), kThreads, 0, (cudaStream_t)stream>>>(
        (const T*)proj, ldp, (T*)ring, slot, pos, seq_row, seq_len, channels, taps);
    return cudaGetLastError();
  });
}

// out[t, h, :] = scale * o / sqrt(mean(o^2) + eps) * w * act(gate), o [tokens, heads, vdim] fp32; w [vdim], or [heads, vdim]
// (per_head); act: silu, or a sigmoid.
IPEX_API int ipex_gated_norm(const float* o, const void* gate, int64_t ldg, const void* w, int per_head, int sigmoid, void* out,
                             int64_t ldo, int tokens, int heads, int vdim, float eps, float scale, int dtype, void* stream) {
  if (tokens < 1 || heads < 1 || vdim < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int64_t rows = (int64_t)tokens * heads;
    const bool vec = vdim % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)o & 15) == 0 &&
                     (((uintptr_t)gate | (uintptr_t)w | (uintptr_t)out) & 7) == 0;
    auto kern = vec ? (sigmoid ? gated_norm_kernel<T, true, true> : gated_norm_kernel<T, true, false>)
                    : (sigmoid ? gated_norm_kernel<T, false, true> : gated_norm_kernel<T, false, false>);
    kern<<<(unsigned)((rows + 7) / 8), kThreads, 0, (cudaStream_t)stream>>>(
        o, (const T*)gate, ldg, (const T*)w, per_head ? vdim : 0, (T*)out, ldo, rows, heads, vdim, eps, scale);
    return cudaGetLastError();
  });
}

// out [tokens, width] = norm(y * silu(z)) * w, the norm over each of `parts` equal parts; y [tokens, width] fp32.
IPEX_API int ipex_gated_group_norm(const float* y, const void* z, int64_t ldz, const void* w, void* out, int64_t ldo,
                                   int tokens, int width, int parts, float eps, int dtype, int pdl, void* stream) {
  if (tokens < 1 || width < 1 || parts < 1 || parts > 65535 || width % parts) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int part = width / parts;
    const bool vec = part % 4 == 0 && ldz % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)y & 15) == 0 &&
                     (((uintptr_t)z | (uintptr_t)w | (uintptr_t)out) & 7) == 0;
    const int packs = vec ? part / 4 : part, threads = packs >= 512 ? kThreads : packs >= 128 ? 128 : packs >= 64 ? 64 : 32;
    auto kern = vec ? gated_group_norm_kernel<T, 4> : gated_group_norm_kernel<T, 1>;
    return launch_kernel(kern, dim3(tokens, parts), dim3(threads), 0, (cudaStream_t)stream, pdl != 0, y, (const T*)z, ldz,
                         (const T*)w, (T*)out, ldo, width, part, eps);
  });
}
