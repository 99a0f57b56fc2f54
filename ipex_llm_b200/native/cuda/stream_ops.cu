// Element-wise and routing kernels of decoders with a 32-bit residual stream, sm_100a: embedding (scaled, with an
// optional bigram table, into one or several streams), RMS norm of the stream into the activation dtype, the joint of a
// block that norms a sublayer's output before it is added, the joint of blocks between which several streams are mixed
// (hyper-connections), the joint of a block whose sublayers' outputs are normed side by side, tanh soft-cap of fp32 logits,
// biases, activations and gated units behind library or packed products, and
// the data movement around a dense expert bank for prompts (choice of experts, slots grouped by expert on the device,
// row gather, gated unit, combination), plus a plain tiled product for sizes the tensor-core kernels do not take and for
// 32-bit models.
#include "common/routing.cuh"
#include "common/utils.cuh"

namespace {

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < (int)(blockDim.x >> 5) ? red[lane] : 0.f;
  return warp_sum(t);
}

// One CTA per token.  The token id is filed in the history [slots, cap] at its position; the bigram row needs the
// token before it, which is either the neighbouring entry of this launch or already in the history.
template <typename T>
__global__ void embed_stream_kernel(const int64_t* __restrict__ tokens, const int* __restrict__ slot,
                                    const int* __restrict__ pos, const int* __restrict__ start, int* history,
                                    int64_t cap, const T* __restrict__ table, const T* __restrict__ bigram,
                                    float* __restrict__ out, int W, int64_t vocab, float scale, int64_t buckets,
                                    int64_t mul_prev, int64_t mul_cur, int copies) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int64_t tok = tokens[t];
  tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
  const int s = slot[t], p = pos[t];
  int64_t row = -1;
  if (bigram != nullptr) {
    row = buckets;
    if (p > start[s]) {
      int64_t prev;
      if (t > 0 && slot[t - 1] == s && pos[t - 1] == p - 1) prev = tokens[t - 1];
      else prev = history[(int64_t)s * cap + p - 1];
      row = (prev * mul_prev + tok * mul_cur) % buckets;
      if (row < 0) row += buckets;
    }
  }
  if (threadIdx.x == 0) history[(int64_t)s * cap + p] = (int)tok;
  const T* e = table + tok * W;
  const T* b = bigram + (row < 0 ? 0 : row) * W;
  float* o = out + (int64_t)t * copies * W;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float v = DT<T>::to_f(e[i]) * scale;
    if (row >= 0) v += DT<T>::to_f(b[i]);
    for (int c = 0; c < copies; ++c) o[(int64_t)c * W + i] = v;
  }
}

template <typename T, typename TW>
__global__ void norm_stream_kernel(const float* __restrict__ x, int64_t ldx, const TW* __restrict__ w,
                                   T* __restrict__ out, int64_t ldo, const int* __restrict__ rows, int K, float eps) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t r = rows != nullptr ? rows[blockIdx.x] : (int)blockIdx.x;
  const float* src = x + r * ldx;
  T* dst = out + (int64_t)blockIdx.x * ldo;
  float s = 0.f;
  const bool v4 = K % 4 == 0 && ldx % 4 == 0;
  if (v4) {
    for (int k = threadIdx.x; k < K / 4; k += blockDim.x) {
      const float4 f = reinterpret_cast<const float4*>(src)[k];
      s += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
    }
  } else {
    for (int k = threadIdx.x; k < K; k += blockDim.x) s = fmaf(src[k], src[k], s);
  }
  s = block_sum(s, red);
  const float inv = 1.0f / sqrtf(s / (float)K + eps);
  if (v4 && ldo % 4 == 0) {
    for (int k = threadIdx.x; k < K / 4; k += blockDim.x) {
      const float4 f = reinterpret_cast<const float4*>(src)[k];
      __align__(16) T o[4];
      o[0] = DT<T>::from_f(f.x * inv * DT<TW>::to_f(w[4 * k]));
      o[1] = DT<T>::from_f(f.y * inv * DT<TW>::to_f(w[4 * k + 1]));
      o[2] = DT<T>::from_f(f.z * inv * DT<TW>::to_f(w[4 * k + 2]));
      o[3] = DT<T>::from_f(f.w * inv * DT<TW>::to_f(w[4 * k + 3]));
      if constexpr (sizeof(T) == 2) reinterpret_cast<uint2*>(dst)[k] = *reinterpret_cast<const uint2*>(o);
      else reinterpret_cast<uint4*>(dst)[k] = *reinterpret_cast<const uint4*>(o);
    }
  } else {
    for (int k = threadIdx.x; k < K; k += blockDim.x) dst[k] = DT<T>::from_f(src[k] * inv * DT<TW>::to_f(w[k]));
  }
}

// x += norm(y) * w_out, and h = norm(x) * w_in in the activation dtype: what stands between two sublayers when the
// first one's output is normed before it is added.  One CTA per row; a thread keeps its part of the row in registers.
constexpr int kJointVec = 4;
template <typename T>
__global__ void add_norm_stream_kernel(float* __restrict__ x, int64_t ldx, const float* __restrict__ y, int64_t ldy,
                                       const float* __restrict__ w_out, const float* __restrict__ w_in,
                                       T* __restrict__ out, int64_t ldo, int K, float eps) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  float* xr = x + (int64_t)blockIdx.x * ldx;
  const float* yr = y + (int64_t)blockIdx.x * ldy;
  T* dst = out + (int64_t)blockIdx.x * ldo;
  const int nt = blockDim.x, tid = threadIdx.x;
  if (K % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && K <= nt * kJointVec * 4) {
    float4 xv[kJointVec], yv[kJointVec];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kJointVec; ++i) {
      const int k = tid + i * nt;
      yv[i] = xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k < K / 4) {
        yv[i] = reinterpret_cast<const float4*>(yr)[k];
        xv[i] = reinterpret_cast<const float4*>(xr)[k];
      }
    }
#pragma unroll
    for (int i = 0; i < kJointVec; ++i)
      s += yv[i].x * yv[i].x + yv[i].y * yv[i].y + yv[i].z * yv[i].z + yv[i].w * yv[i].w;
    s = block_sum(s, red);
    float inv = 1.0f / sqrtf(s / (float)K + eps);
    s = 0.f;
#pragma unroll
    for (int i = 0; i < kJointVec; ++i) {
      const int k = tid + i * nt;
      if (k < K / 4) {
        const float4 w = reinterpret_cast<const float4*>(w_out)[k];
        xv[i].x += yv[i].x * inv * w.x;
        xv[i].y += yv[i].y * inv * w.y;
        xv[i].z += yv[i].z * inv * w.z;
        xv[i].w += yv[i].w * inv * w.w;
        reinterpret_cast<float4*>(xr)[k] = xv[i];
        s += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
      }
    }
    if (out == nullptr) return;
    s = block_sum(s, red);
    inv = 1.0f / sqrtf(s / (float)K + eps);
#pragma unroll
    for (int i = 0; i < kJointVec; ++i) {
      const int k = tid + i * nt;
      if (k < K / 4) {
        const float4 w = reinterpret_cast<const float4*>(w_in)[k];
        const float o[4] = {xv[i].x * inv * w.x, xv[i].y * inv * w.y, xv[i].z * inv * w.z, xv[i].w * inv * w.w};
        if (ldo % 4 == 0) {
          __align__(16) T t[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) t[j] = DT<T>::from_f(o[j]);
          if constexpr (sizeof(T) == 2) reinterpret_cast<uint2*>(dst)[k] = *reinterpret_cast<const uint2*>(t);
          else reinterpret_cast<uint4*>(dst)[k] = *reinterpret_cast<const uint4*>(t);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j) dst[4 * k + j] = DT<T>::from_f(o[j]);
        }
      }
    }
    return;
  }
  float s = 0.f;
  for (int k = tid; k < K; k += nt) s = fmaf(yr[k], yr[k], s);
  s = block_sum(s, red);
  float inv = 1.0f / sqrtf(s / (float)K + eps);
  s = 0.f;
  for (int k = tid; k < K; k += nt) {
    const float v = xr[k] + yr[k] * inv * w_out[k];
    xr[k] = v;
    s = fmaf(v, v, s);
  }
  if (out == nullptr) return;
  s = block_sum(s, red);
  inv = 1.0f / sqrtf(s / (float)K + eps);
  for (int k = tid; k < K; k += nt) dst[k] = DT<T>::from_f(xr[k] * inv * w_in[k]);
}

// x += sum over one or two y of norm(y) * w, and out = x, or norm(x) * w_in, in the activation dtype.  One CTA per row.
struct SidesArgs {
  float* x;
  const float* y[2];    // [n, ldy] or null
  const float* w[2];    // [K]
  const float* w_in;    // [K], or null: out is x itself
  void* out;            // T [n, ldo] or null
  int64_t ldx, ldy, ldo;
  int K;
  float eps;
};

template <typename T>
__global__ void add_sides_kernel(SidesArgs a) {
  __shared__ float red[32], red2[32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, nt = blockDim.x;
  float* x = a.x + (int64_t)blockIdx.x * a.ldx;
  const float* y0 = a.y[0] != nullptr ? a.y[0] + (int64_t)blockIdx.x * a.ldy : nullptr;
  const float* y1 = a.y[1] != nullptr ? a.y[1] + (int64_t)blockIdx.x * a.ldy : nullptr;
  T* out = a.out != nullptr ? reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * a.ldo : nullptr;
  float s0 = 0.f, s1 = 0.f;
  for (int k = tid; k < a.K; k += nt) {
    if (y0 != nullptr) s0 = fmaf(y0[k], y0[k], s0);
    if (y1 != nullptr) s1 = fmaf(y1[k], y1[k], s1);
  }
  if (y0 != nullptr) s0 = 1.0f / sqrtf(block_sum(s0, red) / (float)a.K + a.eps);
  if (y1 != nullptr) s1 = 1.0f / sqrtf(block_sum(s1, red2) / (float)a.K + a.eps);
  float ss = 0.f;
  for (int k = tid; k < a.K; k += nt) {
    float v = x[k];
    if (y0 != nullptr) v = fmaf(y0[k] * s0, a.w[0][k], v);
    if (y1 != nullptr) v = fmaf(y1[k] * s1, a.w[1][k], v);
    if (y0 != nullptr || y1 != nullptr) x[k] = v;
    if (a.w_in != nullptr) ss = fmaf(v, v, ss);
    else if (out != nullptr) out[k] = DT<T>::from_f(v);
  }
  if (a.w_in == nullptr || out == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.K + a.eps);
  for (int k = tid; k < a.K; k += nt) out[k] = DT<T>::from_f(x[k] * inv * a.w_in[k]);      // (what this thread wrote)
}

// Several residual streams x [S, K] per token.  Behind a sublayer with output y all streams are mixed,
// x_t <- sum_s mix[s, t] x_s + w_out[t] y  (y null: they stay), and the next sublayer's input is the norm of
// sum_s w_in[s] x_s.  One CTA per token; with NV > 0 a thread keeps its part of all streams in registers.
struct HyperArgs {
  float* x;             // [n, S, K]
  const float* y;       // [n, ldy] or null
  const float* mix;     // [S, S], from row to column
  const float* w_out;   // [S]
  const float* w_in;    // [S]
  const float* norm;    // [K]
  void* out;            // T [n, ldo]
  int64_t ldy, ldo;
  int S, K;
  float eps;
};
constexpr int kMaxStreams = 16;

template <typename T, int S, int NV>
__global__ void __launch_bounds__(NV == 1 ? 256 : 1024) hyper_joint_kernel(HyperArgs a) {
  __shared__ float red[32];
  __shared__ float s_mix[S * S], s_out[S], s_in[S];
  pdl_launch_dependents();
  const int tid = threadIdx.x, nt = blockDim.x, K4 = a.K / 4;
  if (tid < S) {
    s_in[tid] = a.w_in[tid];
    if (a.y != nullptr) s_out[tid] = a.w_out[tid];
  }
  if (a.y != nullptr && tid < S * S) s_mix[tid] = a.mix[tid];
  pdl_wait();
  __syncthreads();
  float4* x = reinterpret_cast<float4*>(a.x + (int64_t)blockIdx.x * S * a.K);
  float4 u[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = tid + i * nt;
    u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (k >= K4) continue;
    float4 v[S], n[S];
#pragma unroll
    for (int s = 0; s < S; ++s) n[s] = v[s] = x[(int64_t)s * K4 + k];
    if (a.y != nullptr) {
      const float4 y = reinterpret_cast<const float4*>(a.y + (int64_t)blockIdx.x * a.ldy)[k];
#pragma unroll
      for (int t = 0; t < S; ++t) {
        const float o = s_out[t];
        n[t] = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
        for (int s = 0; s < S; ++s) {
          const float m = s_mix[s * S + t];
          n[t].x = fmaf(m, v[s].x, n[t].x);
          n[t].y = fmaf(m, v[s].y, n[t].y);
          n[t].z = fmaf(m, v[s].z, n[t].z);
          n[t].w = fmaf(m, v[s].w, n[t].w);
        }
        x[(int64_t)t * K4 + k] = n[t];
      }
    }
#pragma unroll
    for (int s = 0; s < S; ++s) {
      const float m = s_in[s];
      u[i].x = fmaf(m, n[s].x, u[i].x);
      u[i].y = fmaf(m, n[s].y, u[i].y);
      u[i].z = fmaf(m, n[s].z, u[i].z);
      u[i].w = fmaf(m, n[s].w, u[i].w);
    }
    ss += u[i].x * u[i].x + u[i].y * u[i].y + u[i].z * u[i].z + u[i].w * u[i].w;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)a.K + a.eps);
  T* dst = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * a.ldo;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = tid + i * nt;
    if (k >= K4) continue;
    const float4 w = reinterpret_cast<const float4*>(a.norm)[k];
    __align__(16) T o[4] = {DT<T>::from_f(u[i].x * inv * w.x), DT<T>::from_f(u[i].y * inv * w.y),
                            DT<T>::from_f(u[i].z * inv * w.z), DT<T>::from_f(u[i].w * inv * w.w)};
    if constexpr (sizeof(T) == 2) reinterpret_cast<uint2*>(dst)[k] = *reinterpret_cast<const uint2*>(o);
    else reinterpret_cast<uint4*>(dst)[k] = *reinterpret_cast<const uint4*>(o);
  }
}

template <typename T>
__global__ void hyper_joint_any_kernel(HyperArgs a) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, nt = blockDim.x, S = a.S;
  float* x = a.x + (int64_t)blockIdx.x * S * a.K;
  float ss = 0.f;
  for (int k = tid; k < a.K; k += nt) {
    float v[kMaxStreams], u = 0.f;
    for (int s = 0; s < S; ++s) v[s] = x[(int64_t)s * a.K + k];
    if (a.y != nullptr) {
      const float y = a.y[(int64_t)blockIdx.x * a.ldy + k];
      for (int t = 0; t < S; ++t) {
        float n = a.w_out[t] * y;
        for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], v[s], n);
        x[(int64_t)t * a.K + k] = n;
        u = fmaf(a.w_in[t], n, u);
      }
    } else {
      for (int s = 0; s < S; ++s) u = fmaf(a.w_in[s], v[s], u);
    }
    ss = fmaf(u, u, ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)a.K + a.eps);
  T* dst = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * a.ldo;
  for (int k = tid; k < a.K; k += nt) {
    float u = 0.f;                                  // a thread reads what it wrote itself
    for (int s = 0; s < S; ++s) u = fmaf(a.w_in[s], x[(int64_t)s * a.K + k], u);
    dst[k] = DT<T>::from_f(u * inv * a.norm[k]);
  }
}

template <typename T, int S>
cudaError_t launch_hyper(const HyperArgs& a, int n, bool pdl, cudaStream_t st) {
  const int k4 = a.K / 4;
  if (k4 <= 256) return launch_kernel(hyper_joint_kernel<T, S, 1>, dim3(n), dim3((k4 + 31) / 32 * 32), 0, st, pdl, a);
  const int half = (k4 + 1) / 2, threads = (half + 31) / 32 * 32;
  return launch_kernel(hyper_joint_kernel<T, S, 2>, dim3(n), dim3(threads < 256 ? 256 : threads), 0, st, pdl, a);
}

// y += bias, row by row
template <typename TY, typename T>
__global__ void bias_rows_kernel(TY* __restrict__ y, int64_t ldy, const T* __restrict__ bias, int N) {
  TY* r = y + (int64_t)blockIdx.x * ldy;
  for (int n = threadIdx.x; n < N; n += blockDim.x) r[n] = DT<TY>::from_f(DT<TY>::to_f(r[n]) + DT<T>::to_f(bias[n]));
}

// out[r, i] = act(gate + bias) * (up + bias) from a row of 2 I products, act gelu_tanh (3), silu (4) or the clamped unit (5);
// interleaved: gate and up alternate in blocks of eight
template <typename TY, typename T, int ACT>
__global__ void glu_products_kernel(const TY* __restrict__ gu, int64_t ld, const T* __restrict__ bias,
                                     T* __restrict__ out, int64_t ldo, int I, int interleaved, float limit, float alpha) {
  const TY* r = gu + (int64_t)blockIdx.x * ld;
  for (int i = threadIdx.x; i < I; i += blockDim.x) {
    const int g = interleaved ? (i >> 3) * 16 + (i & 7) : i, u = interleaved ? g + 8 : I + i;
    const float bg = bias != nullptr ? DT<T>::to_f(bias[g]) : 0.f, bu = bias != nullptr ? DT<T>::to_f(bias[u]) : 0.f;
    const float z = DT<TY>::to_f(r[g]) + bg;
    const float v = DT<TY>::to_f(r[u]) + bu;
    float y;
    if constexpr (ACT == 5) {
      const float g1 = fminf(z, limit);
      y = g1 / (1.0f + expf(-alpha * g1)) * (fminf(fmaxf(v, -limit), limit) + 1.0f);
    } else {
      y = (ACT == 4 ? silu(z) : gelu_tanh(z)) * v;
    }
    out[(int64_t)blockIdx.x * ldo + i] = DT<T>::from_f(y);
  }
}

// columns [from, N) of y in place: act 1 squared relu; 6 gelu_tanh times row ids[r] of mul
template <typename TY, typename T>
__global__ void act_rows_kernel(TY* __restrict__ y, int64_t ldy, int N, int from, int act, const T* __restrict__ mul,
                                int64_t ldm, int64_t mul_rows, const int64_t* __restrict__ ids) {
  TY* r = y + (int64_t)blockIdx.x * ldy;
  const int64_t row = act == 6 ? min(max(ids[blockIdx.x], (int64_t)0), mul_rows - 1) : 0;
  for (int n = from + threadIdx.x; n < N; n += blockDim.x) {
    const float v = DT<TY>::to_f(r[n]);
    r[n] = DT<TY>::from_f(act == 6 ? gelu_tanh(v) * DT<T>::to_f(mul[row * ldm + n]) : v > 0.f ? v * v : 0.f);
  }
}

__global__ void softcap_kernel(float* x, int64_t n, float cap) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

// x += y for a row-major y of the activation dtype (packed-weight projections, whose kernels write 16 bits)
template <typename T>
__global__ void add_stream_kernel(float* __restrict__ x, const T* __restrict__ y, int64_t n) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] += DT<T>::to_f(y[i]);
}

template <typename T>
__global__ void relu2_kernel(T* x, int64_t n) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) {
    const float v = fmaxf(DT<T>::to_f(x[i]), 0.f);
    x[i] = DT<T>::from_f(v * v);
  }
}

// ---------------------------------------------------------------------------------------------- routing for prompts
// fp32 router logits [tokens, E] -> the k largest sigmoid scores and their experts; a warp per token.
__global__ void sigmoid_topk_kernel(const float* __restrict__ logits, int64_t ld, float* __restrict__ w,
                                    int64_t* __restrict__ idx, int tokens, int E, int k) {
  extern __shared__ float sh[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wpb = blockDim.x >> 5;
  const int t = blockIdx.x * wpb + warp;
  if (t >= tokens) return;
  float* sc = sh + (size_t)warp * E;
  for (int e = lane; e < E; e += 32) sc[e] = 1.0f / (1.0f + expf(-logits[(int64_t)t * ld + e]));
  __syncwarp();
  for (int r = 0; r < k; ++r) {
    float best = -1.f;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32)
      if (sc[e] > best) { best = sc[e]; bi = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (bi >= E) { bi = 0; best = 0.f; }
    if (lane == 0) {
      w[(int64_t)t * k + r] = best;
      idx[(int64_t)t * k + r] = bi;
      sc[bi] = -2.f;
    }
    __syncwarp();
  }
}

// fp32 router logits [tokens, E (+ 1)] -> weights and experts (softmax_grouped_topk) in rows of ldk; a warp per token.  bias:
// [E] or null, added to the logits.  gate: the logit behind the experts' becomes gate[t] = sigmoid.  always: choice k is expert
// E with weight 1.
__global__ void softmax_topk_kernel(const float* __restrict__ logits, int64_t ld, const float* __restrict__ bias,
                                    float* __restrict__ w, int64_t* __restrict__ idx, int ldk, float* __restrict__ gate,
                                    int always, int tokens, int E, int groups, int keep, int k, float scale) {
  extern __shared__ float sh[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wpb = blockDim.x >> 5;
  const int t = blockIdx.x * wpb + warp;
  if (t >= tokens) return;
  float* sc = sh + (size_t)warp * (E + groups);
  const float* row = logits + (int64_t)t * ld;
  for (int e = lane; e < E; e += 32) sc[e] = bias != nullptr ? row[e] + bias[e] : row[e];
  if (gate != nullptr && lane == 0) gate[t] = 1.0f / (1.0f + expf(-row[E]));
  __syncwarp();
  if (always && lane == 0) {
    w[(int64_t)t * ldk + k] = 1.f;
    idx[(int64_t)t * ldk + k] = E;
  }
  softmax_grouped_topk(sc, sc + E, E, groups, keep, k, scale, w + (int64_t)t * ldk, idx + (int64_t)t * ldk, lane);
}

// (token, choice) slots grouped by expert, one CTA: order[pos] = slot, inverse[slot] = pos, ranges[e] = (first, count).
// The order inside an expert is arbitrary (every row is computed on its own).
__global__ void __launch_bounds__(1024) group_slots_kernel(const int64_t* __restrict__ ids, int slots, int E,
                                                           int* __restrict__ order, int* __restrict__ inverse,
                                                           int* __restrict__ ranges) {
  extern __shared__ int cnt[];        // [E] counts, then next free position
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int s = threadIdx.x; s < slots; s += blockDim.x) atomicAdd(&cnt[(int)ids[s]], 1);
  __syncthreads();
  if (threadIdx.x < 32) {             // exclusive prefix over the experts, one warp
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int c = e < E ? cnt[e] : 0;
      int p = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, p, o);
        if ((int)threadIdx.x >= o) p += v;
      }
      if (e < E) {
        ranges[2 * e] = run + p - c;
        ranges[2 * e + 1] = c;
        cnt[e] = run + p - c;
      }
      run += __shfl_sync(0xffffffffu, p, 31);
    }
  }
  __syncthreads();
  for (int s = threadIdx.x; s < slots; s += blockDim.x) {
    const int p = atomicAdd(&cnt[(int)ids[s]], 1);
    order[p] = s;
    inverse[s] = p;
  }
}

// xs[pos] = x[order[pos] / k], ws[pos] = w[order[pos]]
template <typename T>
__global__ void gather_slots_kernel(const T* __restrict__ x, const float* __restrict__ w, const int* __restrict__ order,
                                    T* __restrict__ xs, float* __restrict__ ws, int K, int k) {
  const int p = blockIdx.x, s = order[p];
  const T* src = x + (int64_t)(s / k) * K;
  T* dst = xs + (int64_t)p * K;
  if (K % (16 / (int)sizeof(T)) == 0) {
    const int nv = K * (int)sizeof(T) / 16;
    for (int i = threadIdx.x; i < nv; i += blockDim.x)
      reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
  } else {
    for (int i = threadIdx.x; i < K; i += blockDim.x) dst[i] = src[i];
  }
  if (threadIdx.x == 0) ws[p] = w[s];
}

// y = g * sigmoid(alpha g) * (u + 1) with g = min(ws * gate, limit), u = clamp(ws * up, +-limit); gu fp32 [rows, 2I]
template <typename T>
__global__ void glu_rows_kernel(const float* __restrict__ gu, const float* __restrict__ ws, T* __restrict__ y, int I,
                                float limit, float alpha, int interleaved) {
  const int r = blockIdx.x;
  const float w = ws[r];
  const float* row = gu + (int64_t)r * 2 * I;
  for (int i = threadIdx.x; i < I; i += blockDim.x) {
    const int gi = interleaved ? (i >> 4) * 32 + (i & 15) : i;
    const int ui = interleaved ? gi + 16 : I + i;
    const float g = fminf(row[gi] * w, limit);
    const float u = fminf(fmaxf(row[ui] * w, -limit), limit);
    y[(int64_t)r * I + i] = DT<T>::from_f(g / (1.0f + expf(-alpha * g)) * (u + 1.0f));
  }
}

// residual[t] += sum_j y[inverse[t * k + j]]
template <typename T>
__global__ void combine_slots_kernel(const T* __restrict__ y, const int* __restrict__ inverse,
                                     float* __restrict__ residual, int N, int k) {
  const int t = blockIdx.x;
  float* o = residual + (int64_t)t * N;
  for (int n = threadIdx.x; n < N; n += blockDim.x) {
    float s = 0.f;
    for (int j = 0; j < k; ++j) s += DT<T>::to_f(y[(int64_t)inverse[(int64_t)t * k + j] * N + n]);
    o[n] += s;
  }
}

// out[t] = gate[t] * out[t] (gate null: 0, or with `add` 1) + sum_j w[t, j] y[inverse[t * k + j]]
template <typename T>
__global__ void combine_weighted_kernel(const T* __restrict__ y, const int* __restrict__ inverse,
                                        const float* __restrict__ w, const float* __restrict__ gate,
                                        float* __restrict__ out, int N, int k, int add) {
  const int t = blockIdx.x;
  float* o = out + (int64_t)t * N;
  const bool keep = gate != nullptr || add;
  const float g = gate != nullptr ? gate[t] : 1.f;
  constexpr int VN = 16 / (int)sizeof(T);
  if (N % VN == 0) {
    for (int n = threadIdx.x * VN; n < N; n += blockDim.x * VN) {
      float s[VN];
#pragma unroll
      for (int i = 0; i < VN; i += 4) {
        const float4 f = keep ? *reinterpret_cast<const float4*>(o + n + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        s[i] = g * f.x; s[i + 1] = g * f.y; s[i + 2] = g * f.z; s[i + 3] = g * f.w;
      }
      for (int j = 0; j < k; ++j) {
        const float wj = w[(int64_t)t * k + j];
        const uint4 raw = *reinterpret_cast<const uint4*>(y + (int64_t)inverse[(int64_t)t * k + j] * N + n);
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < VN; ++i) s[i] = fmaf(wj, DT<T>::to_f(e[i]), s[i]);
      }
#pragma unroll
      for (int i = 0; i < VN; i += 4) *reinterpret_cast<float4*>(o + n + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
    }
    return;
  }
  for (int n = threadIdx.x; n < N; n += blockDim.x) {
    float s = keep ? g * o[n] : 0.f;
    for (int j = 0; j < k; ++j)
      s = fmaf(w[(int64_t)t * k + j], DT<T>::to_f(y[(int64_t)inverse[(int64_t)t * k + j] * N + n]), s);
    o[n] = s;
  }
}

// ------------------------------------------------------------------------------------------- plain tiled product
// out[m, n] (fp32 or T) = sum_k x[m, k] w[n, k], 64 x 64 tiles, fp32 FMAs; with ranges, group g multiplies its rows
// [ranges[g][0], + ranges[g][1]) of x by weight matrix g.
template <typename T, typename TO>
__global__ void __launch_bounds__(256) gemm_plain_kernel(const T* __restrict__ x, const T* __restrict__ w,
                                                         TO* __restrict__ out, const int* __restrict__ ranges, int M,
                                                         int N, int K) {
  __shared__ float sa[16][65], sb[16][65];
  int row0 = 0;
  if (ranges != nullptr) {
    row0 = ranges[2 * blockIdx.z];
    M = ranges[2 * blockIdx.z + 1];
    w += (int64_t)blockIdx.z * N * K;
  }
  const int n0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  for (int m0 = blockIdx.y * 64; m0 < M; m0 += gridDim.y * 64) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += 16) {
      for (int i = threadIdx.x; i < 1024; i += 256) {
        const int kk = i & 15, r = i >> 4;
        const int k = k0 + kk;
        sa[kk][r] = (m0 + r < M && k < K) ? DT<T>::to_f(x[(int64_t)(row0 + m0 + r) * K + k]) : 0.f;
        sb[kk][r] = (n0 + r < N && k < K) ? DT<T>::to_f(w[(int64_t)(n0 + r) * K + k]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int kk = 0; kk < 16; ++kk) {
        float av[4], bv[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) { av[i] = sa[kk][ty + 16 * i]; bv[i] = sb[kk][tx + 16 * i]; }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int m = m0 + ty + 16 * i, n = n0 + tx + 16 * j;
        if (m < M && n < N) out[(int64_t)(row0 + m) * N + n] = DT<TO>::from_f(acc[i][j]);
      }
  }
}

}  // namespace

// out[t] = table[token] * scale (+ bigram row), fp32, `copies` times behind one another.  history: int32 [slots, cap]; start: int32 [slots], the position
// of each sequence's first token.  bigram may be null (buckets etc. are ignored then).
IPEX_API int ipex_embed_stream(const int64_t* tokens, const int* slot, const int* pos, const int* start, int* history,
                               int64_t cap, const void* table, const void* bigram, float* out, int n, int W,
                               int64_t vocab, float scale, int64_t buckets, int64_t mul_prev, int64_t mul_cur, int copies,
                               int dtype, int pdl, void* stream) {
  if (n < 1 || W < 1 || copies < 1 || (bigram != nullptr && buckets < 1)) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return launch_kernel(embed_stream_kernel<T>, dim3(n), dim3(256), 0, (cudaStream_t)stream, pdl != 0, tokens, slot,
                         pos, start, history, cap, (const T*)table, (const T*)bigram, out, W, vocab, scale, buckets,
                         mul_prev, mul_cur, copies);
  });
}

// out[i] = RMS norm of row rows[i] (or i) of the fp32 stream, in the activation dtype; the weight has that dtype too, or
// is fp32 (w_f32).
IPEX_API int ipex_norm_stream(const float* x, int64_t ldx, const void* w, int w_f32, void* out, int64_t ldo,
                              const int* rows, int n, int K, float eps, int dtype, int pdl, void* stream) {
  if (n < 1 || K < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (w_f32)
      return launch_kernel(norm_stream_kernel<T, float>, dim3(n), dim3(256), 0, (cudaStream_t)stream, pdl != 0, x, ldx,
                           (const float*)w, (T*)out, ldo, rows, K, eps);
    return launch_kernel(norm_stream_kernel<T, T>, dim3(n), dim3(256), 0, (cudaStream_t)stream, pdl != 0, x, ldx,
                         (const T*)w, (T*)out, ldo, rows, K, eps);
  });
}

// x [n, K] += RMS norm of y times w_out; out (may be null) = RMS norm of the new x times w_in.  Weights fp32, 16-byte
// aligned like x and y.
IPEX_API int ipex_add_norm_stream(float* x, int64_t ldx, const float* y, int64_t ldy, const float* w_out,
                                  const float* w_in, void* out, int64_t ldo, int n, int K, float eps, int dtype, int pdl,
                                  void* stream) {
  if (n < 1 || K < 1 || (out != nullptr && w_in == nullptr)) return (int)cudaErrorInvalidValue;
  if (((uintptr_t)x | (uintptr_t)y | (uintptr_t)w_out | (uintptr_t)w_in | (uintptr_t)out) & 15)
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int threads = K <= 2048 ? 256 : K <= 4096 ? 512 : 1024;
    return launch_kernel(add_norm_stream_kernel<T>, dim3(n), dim3(threads), 0, (cudaStream_t)stream, pdl != 0, x, ldx, y,
                         ldy, w_out, w_in, (T*)out, ldo, K, eps);
  });
}

// x [n, K] += norm(y0) * w0 + norm(y1) * w1 (y0, y1 may be null; row stride ldy); out (may be null) = x in the activation
// dtype, or norm(x) * w_in.  Weights fp32.
IPEX_API int ipex_add_sides(float* x, int64_t ldx, const float* y0, const float* w0, const float* y1, const float* w1,
                            int64_t ldy, const float* w_in, void* out, int64_t ldo, int n, int K, float eps, int dtype, int pdl,
                            void* stream) {
  if (n < 1 || K < 1 || (y0 != nullptr && w0 == nullptr) || (y1 != nullptr && w1 == nullptr)) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const SidesArgs a = {x, {y0, y1}, {w0, w1}, w_in, out, ldx, ldy, ldo, K, eps};
    const int threads = K <= 512 ? 128 : K <= 2048 ? 256 : K <= 4096 ? 512 : 1024;
    return launch_kernel(add_sides_kernel<T>, dim3(n), dim3(threads), 0, (cudaStream_t)stream, pdl != 0, a);
  });
}

// Columns [from, N) of y [n, N] (the activation dtype, or fp32) in place: act 1 squared relu; 6 gelu_tanh times the row ids[i] of
// mul [mul_rows, ldm].
IPEX_API int ipex_act_rows(void* y, int64_t ldy, int y_f32, int n, int N, int from, int act, const void* mul, int64_t ldm,
                           int64_t mul_rows, const int64_t* ids, int dtype, void* stream) {
  if (n < 1 || N < 1 || from < 0 || (act != 1 && act != 6) || (act == 6 && (mul == nullptr || ids == nullptr || mul_rows < 1)))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    cudaStream_t st = (cudaStream_t)stream;
    if (y_f32) act_rows_kernel<float, T><<<n, 256, 0, st>>>((float*)y, ldy, N, from, act, (const T*)mul, ldm, mul_rows, ids);
    else act_rows_kernel<T, T><<<n, 256, 0, st>>>((T*)y, ldy, N, from, act, (const T*)mul, ldm, mul_rows, ids);
    return cudaGetLastError();
  });
}

// y [n, N] (the bias's dtype, or fp32) += bias
IPEX_API int ipex_bias_rows(void* y, int64_t ldy, int y_f32, const void* bias, int n, int N, int dtype, void* stream) {
  if (n < 1 || N < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (y_f32) bias_rows_kernel<float, T><<<n, 256, 0, (cudaStream_t)stream>>>((float*)y, ldy, (const T*)bias, N);
    else bias_rows_kernel<T, T><<<n, 256, 0, (cudaStream_t)stream>>>((T*)y, ldy, (const T*)bias, N);
    return cudaGetLastError();
  });
}

// out [n, I] = act(gate + bias) * (up + bias) of gu [n, 2 I] (the activation dtype, or fp32); act: see glu_products_kernel
IPEX_API int ipex_glu_rows(const void* gu, int64_t ld, int gu_f32, const void* bias, void* out, int64_t ldo, int n, int I,
                           int interleaved, int act, float limit, float alpha, int dtype, void* stream) {
  if (n < 1 || I < 1 || (interleaved && I % 8 != 0) || act < 3 || act > 5) return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (gu_f32) {
      auto kern = act == 5 ? glu_products_kernel<float, T, 5> : act == 4 ? glu_products_kernel<float, T, 4> : glu_products_kernel<float, T, 3>;
      kern<<<n, 256, 0, st>>>((const float*)gu, ld, (const T*)bias, (T*)out, ldo, I, interleaved, limit, alpha);
    } else {
      auto kern = act == 5 ? glu_products_kernel<T, T, 5> : act == 4 ? glu_products_kernel<T, T, 4> : glu_products_kernel<T, T, 3>;
      kern<<<n, 256, 0, st>>>((const T*)gu, ld, (const T*)bias, (T*)out, ldo, I, interleaved, limit, alpha);
    }
    return cudaGetLastError();
  });
}

// Behind a sublayer of a decoder with S residual streams: see HyperArgs.  y null: the streams stay as they are.
IPEX_API int ipex_hyper_joint(float* x, const float* y, int64_t ldy, const float* mix, const float* w_out,
                              const float* w_in, const float* norm, void* out, int64_t ldo, int n, int S, int K, float eps,
                              int dtype, int pdl, void* stream) {
  if (n < 1 || S < 1 || S > kMaxStreams || K < 1 || x == nullptr || w_in == nullptr || norm == nullptr || out == nullptr ||
      (y != nullptr && (mix == nullptr || w_out == nullptr)))
    return (int)cudaErrorInvalidValue;
  HyperArgs a = {x, y, mix, w_out, w_in, norm, out, ldy, ldo, S, K, eps};
  const bool vec = K % 4 == 0 && K <= 8192 && ldo % 4 == 0 && ldy % 4 == 0 &&
                   (((uintptr_t)x | (uintptr_t)y | (uintptr_t)norm | (uintptr_t)out) & 15) == 0;
  cudaStream_t st = (cudaStream_t)stream;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (vec && S == 1) return launch_hyper<T, 1>(a, n, pdl != 0, st);
    if (vec && S == 2) return launch_hyper<T, 2>(a, n, pdl != 0, st);
    if (vec && S == 3) return launch_hyper<T, 3>(a, n, pdl != 0, st);
    if (vec && S == 4) return launch_hyper<T, 4>(a, n, pdl != 0, st);
    return launch_kernel(hyper_joint_any_kernel<T>, dim3(n), dim3(256), 0, st, pdl != 0, a);
  });
}

IPEX_API int ipex_softcap_f32(float* x, int64_t n, float cap, void* stream) {
  if (n < 1 || !(cap > 0.f)) return (int)cudaErrorInvalidValue;
  softcap_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, n, cap);
  return (int)cudaGetLastError();
}

IPEX_API int ipex_add_stream(float* x, const void* y, int64_t n, int dtype, void* stream) {
  if (n < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    add_stream_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, (const T*)y, n);
    return cudaGetLastError();
  });
}

IPEX_API int ipex_relu2_inplace(void* x, int64_t n, int dtype, void* stream) {
  if (n < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    relu2_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>((T*)x, n);
    return cudaGetLastError();
  });
}

IPEX_API int ipex_moe_sigmoid_topk(const float* logits, int64_t ld, float* w, int64_t* idx, int tokens, int E, int k,
                                   void* stream) {
  if (tokens < 1 || E < 1 || E > 3000 || k < 1 || k > E) return (int)cudaErrorInvalidValue;
  sigmoid_topk_kernel<<<(tokens + 3) / 4, 128, (size_t)4 * E * sizeof(float), (cudaStream_t)stream>>>(
      logits, ld, w, idx, tokens, E, k);
  return (int)cudaGetLastError();
}

// logits [tokens, E] (with `gate`, E + 1) -> weights and experts [tokens, k]: soft-max, the `keep` best of `groups` equal
// groups, the k largest, divided by their sum and times scale; gate [tokens] (may be null): sigmoid of the last logit.  bias
// [E] (may be null) is added to the logits.  w and idx have rows of ldk; always: choice k is expert E, weight 1.
IPEX_API int ipex_moe_softmax_grouped_topk(const float* logits, int64_t ld, const float* bias, float* w, int64_t* idx, int ldk,
                                           float* gate, int always, int tokens, int E, int groups, int keep, int k,
                                           float scale, int pdl, void* stream) {
  if (tokens < 1 || E < 1 || E > 2500 || k < 1 || k > E || groups < 1 || E % groups || keep < 1 || keep > groups ||
      k > E / groups * keep || ldk < k + (always != 0))
    return (int)cudaErrorInvalidValue;
  return (int)launch_kernel(softmax_topk_kernel, dim3((tokens + 3) / 4), dim3(128), (size_t)4 * (E + groups) * sizeof(float),
                            (cudaStream_t)stream, pdl != 0, logits, ld, bias, w, idx, ldk, gate, always, tokens, E, groups, keep, k,
                            scale);
}

// Expert ids must lie in [0, E).
IPEX_API int ipex_moe_group_slots(const int64_t* ids, int slots, int E, int* order, int* inverse, int* ranges,
                                  void* stream) {
  if (slots < 1 || E < 1 || E > 12000) return (int)cudaErrorInvalidValue;
  group_slots_kernel<<<1, 1024, (size_t)E * sizeof(int), (cudaStream_t)stream>>>(ids, slots, E, order, inverse, ranges);
  return (int)cudaGetLastError();
}

IPEX_API int ipex_moe_gather_slots(const void* x, const float* w, const int* order, void* xs, float* ws, int slots,
                                   int K, int k, int dtype, void* stream) {
  if (slots < 1 || K < 1 || k < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    gather_slots_kernel<T><<<slots, 128, 0, (cudaStream_t)stream>>>((const T*)x, w, order, (T*)xs, ws, K, k);
    return cudaGetLastError();
  });
}

IPEX_API int ipex_moe_glu_from_gu(const float* gu, const float* ws, void* y, int rows, int I, float limit, float alpha,
                                  int interleaved, int dtype, void* stream) {
  if (rows < 1 || I < 1 || (interleaved && I % 16 != 0)) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    glu_rows_kernel<T><<<rows, 128, 0, (cudaStream_t)stream>>>(gu, ws, (T*)y, I, limit, alpha, interleaved);
    return cudaGetLastError();
  });
}

IPEX_API int ipex_moe_combine_slots(const void* y, const int* inverse, float* residual, int tokens, int N, int k,
                                    int dtype, void* stream) {
  if (tokens < 1 || N < 1 || k < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    combine_slots_kernel<T><<<tokens, 256, 0, (cudaStream_t)stream>>>((const T*)y, inverse, residual, N, k);
    return cudaGetLastError();
  });
}

// out [tokens, N] fp32 = gate * out (gate null: 0, or with `add` 1) + sum_j w[t, j] y[inverse[t k + j]]
IPEX_API int ipex_moe_combine_weighted(const void* y, const int* inverse, const float* w, const float* gate, float* out,
                                       int tokens, int N, int k, int add, int dtype, void* stream) {
  if (tokens < 1 || N < 1 || k < 1 || (((uintptr_t)y | (uintptr_t)out) & 15)) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    combine_weighted_kernel<T><<<tokens, 256, 0, (cudaStream_t)stream>>>((const T*)y, inverse, w, gate, out, N, k, add);
    return cudaGetLastError();
  });
}

// out = x . w^T with contiguous operands; ranges (device, [groups][2]) may be null (groups = 1).  out_f32: fp32 output.
IPEX_API int ipex_gemm_plain(const void* x, const void* w, void* out, const int* ranges, int groups, int M, int N, int K,
                             int out_f32, int dtype, void* stream) {
  if (M < 1 || N < 1 || K < 1 || groups < 1 || groups > 65535) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int mt = (M + 63) / 64;
    dim3 grid((N + 63) / 64, mt < 1024 ? mt : 1024, groups);
    cudaStream_t st = (cudaStream_t)stream;
    if (out_f32)
      gemm_plain_kernel<T, float><<<grid, 256, 0, st>>>((const T*)x, (const T*)w, (float*)out, ranges, M, N, K);
    else
      gemm_plain_kernel<T, T><<<grid, 256, 0, st>>>((const T*)x, (const T*)w, (T*)out, ranges, M, N, K);
    return cudaGetLastError();
  });
}
