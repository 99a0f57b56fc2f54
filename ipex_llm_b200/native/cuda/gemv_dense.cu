// Few-row products with dense 16-bit or 32-bit weights for decoders that keep a 32-bit residual stream, sm_100a.
//
//   gemv_rows    y[M <= 8, N] = act( x . W[N, K]^T )   with x either activations in the weight dtype or the fp32
//                residual stream, RMS-normed while it is staged in shared memory; the result (plus a bias) goes out in
//                the weight dtype, is added to an fp32 residual, or leaves as fp32 with an optional tanh soft-cap
//                (logits); gate and up rows may be joined to gelu_tanh(gate) * up, silu(gate) * up or a clamped unit, results
//                to gelu_tanh(.) * the token's row of a table, and the rows of a second matrix may ride along with fp32
//                results (gates of a recurrence beside its projections)
//   moe_router   norm + router scores in fp32 + sigmoid + top-k of one token per CTA; or, from finished rows, soft-max
//                scores, group-limited top-k with renormalised weights, and the gate of a shared expert
//   moe_glu      per (token, choice) slot: gated unit of the chosen expert - clamped (with the routing weight applied to the
//                expert's input, or not), or silu; a shared expert of another size is one more choice
//   moe_down     residual[t] += sum over the token's choices of down_e(y), weighted or not, or fp32 rows of the weighted sum
//
// All products are fp32 FMAs over 16-byte weight loads: with up to eight rows the weights are the traffic, and eight
// rows of FMAs still fit under the memory time.  A warp owns R weight rows and walks K in steps of 32 vectors with
// several loads in flight per lane.  With programmatic dependent launch the rows a warp touches first are pulled
// into L2 while the previous kernel drains.
#include "common/routing.cuh"
#include "common/utils.cuh"

namespace {

constexpr int kThreads = 512;
constexpr int kWarps = kThreads / 32;

template <typename T> struct Vec {
  static constexpr int n = 16 / sizeof(T);
};

template <typename T>
__device__ __forceinline__ void unpack(const uint4& v, float (&f)[Vec<T>::n]) {
  if constexpr (sizeof(T) == 4) {
    f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
  } else if constexpr (std::is_same<T, __nv_bfloat16>::value) {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
  } else {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 t = __half22float2(*reinterpret_cast<const __half2*>(&w[i]));
      f[2 * i] = t.x;
      f[2 * i + 1] = t.y;
    }
  }
}

// acc[m][r] += sum_k x[m][k] * w[r][k]; x in shared memory (row stride kp elements, zero-filled past K), weight rows
// in global memory.  `vec`: K is a multiple of the vector width and the rows are 16-byte aligned.
template <typename T, int M, int R>
__device__ __forceinline__ void dot_rows(const T* const (&w)[R], const T* sx, int kp, int K, bool vec, int lane,
                                         float (&acc)[M][R]) {
  constexpr int VN = Vec<T>::n;
  constexpr int U = R >= 4 ? 2 : 4;
  if (vec) {
    const int nv = K / VN;
    for (int v0 = 0; v0 < nv; v0 += 32 * U) {
      uint4 raw[U][R];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int v = v0 + u * 32 + lane;
#pragma unroll
        for (int r = 0; r < R; ++r)
          raw[u][r] = v < nv ? ldg_nc_v4(reinterpret_cast<const uint4*>(w[r]) + v) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int v = v0 + u * 32 + lane;
        if (v >= nv) break;
        float wf[R][VN];
#pragma unroll
        for (int r = 0; r < R; ++r) unpack<T>(raw[u][r], wf[r]);
#pragma unroll
        for (int m = 0; m < M; ++m) {
          float xf[VN];
          unpack<T>(*reinterpret_cast<const uint4*>(sx + (size_t)m * kp + v * VN), xf);
#pragma unroll
          for (int r = 0; r < R; ++r)
#pragma unroll
            for (int i = 0; i < VN; ++i) acc[m][r] = fmaf(xf[i], wf[r][i], acc[m][r]);
        }
      }
    }
  } else {
    for (int k = lane; k < K; k += 32) {
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float wv = DT<T>::to_f(w[r][k]);
#pragma unroll
        for (int m = 0; m < M; ++m) acc[m][r] = fmaf(DT<T>::to_f(sx[(size_t)m * kp + k]), wv, acc[m][r]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int r = 0; r < R; ++r) acc[m][r] = warp_sum(acc[m][r]);
}

// block-wide sum (every thread gets it)
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < (int)(blockDim.x >> 5) ? red[lane] : 0.f;
  return warp_sum(t);
}

// Stage `rows` rows: plain copy of T rows, or fp32 rows converted (x_f32) or RMS-normed.  Zero fill up to kp.  Whole block;
// `red` holds one float per warp.
template <typename T>
__device__ __forceinline__ void stage_rows(T* sx, int kp, const void* x, int64_t ldx, const T* norm_w, float eps,
                                           int rows, int K, float* red, bool x_f32 = false) {
  constexpr int VN = Vec<T>::n;
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int m = 0; m < rows; ++m)
    for (int k = K + threadIdx.x; k < kp; k += blockDim.x) sx[(size_t)m * kp + k] = DT<T>::from_f(0.f);
  if (norm_w == nullptr && x_f32) {
    for (int m = 0; m < rows; ++m) {
      const float* src = reinterpret_cast<const float*>(x) + (int64_t)m * ldx;
      for (int k = threadIdx.x; k < K; k += blockDim.x) sx[(size_t)m * kp + k] = DT<T>::from_f(src[k]);
    }
    __syncthreads();
    return;
  }
  if (norm_w == nullptr) {
    for (int m = 0; m < rows; ++m) {
      T* dst = sx + (size_t)m * kp;
      const T* src = reinterpret_cast<const T*>(x) + (int64_t)m * ldx;
      if (K % VN == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
        for (int v = threadIdx.x; v < K / VN; v += blockDim.x)
          reinterpret_cast<uint4*>(dst)[v] = reinterpret_cast<const uint4*>(src)[v];
      } else {
        for (int k = threadIdx.x; k < K; k += blockDim.x) dst[k] = src[k];
      }
    }
    __syncthreads();
    return;
  }
  // `per` warps share a row: the sums of all rows meet in one barrier
  const int per = rows >= warps ? 1 : warps / rows;
  for (int m0 = 0; m0 < rows; m0 += warps / per) {
    const int m = m0 + warp / per, sub = warp % per;
    const bool on = m < rows && warp < warps / per * per;
    const float* src = reinterpret_cast<const float*>(x) + (int64_t)(on ? m : 0) * ldx;
    const bool v4 = K % 4 == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0;
    float s = 0.f;
    if (on) {
      if (v4) {
#pragma unroll 4
        for (int k = sub * 32 + lane; k < K / 4; k += per * 32) {
          const float4 f = reinterpret_cast<const float4*>(src)[k];
          s += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
        }
      } else {
        for (int k = sub * 32 + lane; k < K; k += per * 32) s = fmaf(src[k], src[k], s);
      }
    }
    s = warp_sum(s);
    __syncthreads();
    if (lane == 0) red[warp] = s;
    __syncthreads();
    if (on) {
      s = 0.f;
      for (int i = 0; i < per; ++i) s += red[warp / per * per + i];
      const float inv = 1.0f / sqrtf(s / (float)K + eps);
      T* dst = sx + (size_t)m * kp;
      if (v4) {
#pragma unroll 4
        for (int k = sub * 32 + lane; k < K / 4; k += per * 32) {
          const float4 f = reinterpret_cast<const float4*>(src)[k];
          dst[4 * k] = DT<T>::from_f(f.x * inv * DT<T>::to_f(norm_w[4 * k]));
          dst[4 * k + 1] = DT<T>::from_f(f.y * inv * DT<T>::to_f(norm_w[4 * k + 1]));
          dst[4 * k + 2] = DT<T>::from_f(f.z * inv * DT<T>::to_f(norm_w[4 * k + 2]));
          dst[4 * k + 3] = DT<T>::from_f(f.w * inv * DT<T>::to_f(norm_w[4 * k + 3]));
        }
      } else {
        for (int k = sub * 32 + lane; k < K; k += per * 32)
          dst[k] = DT<T>::from_f(src[k] * inv * DT<T>::to_f(norm_w[k]));
      }
    }
  }
  __syncthreads();
}

struct GemvRowsArgs {
  const void* w;         // [N, K], row stride ldw
  const void* x;         // T [M, K] or fp32 [M, K] (norm_w != null or x_f32), row stride ldx
  const void* norm_w;    // T [K] or null
  void* out;             // out_mode 0: T [M, N]; 1: fp32, accumulated into; 2: fp32 written (soft-capped)
  int64_t ldw, ldx, ldo;
  float eps, softcap;
  int M, N, K, kp;
  int out_mode, act;     // act 1: square of relu; 3 / 4 / 5: gelu_tanh / silu(gate) * up / clamped unit, N / 2 columns come
                         // out; 6: gelu_tanh times the token's row of `mul`
  int vec;
  const void* bias;      // T [N] or null
  const void* w2;        // rows N1 .. N (row stride ldw), or null (then N1 = N)
  float* out2;           // ... and their results, fp32
  int64_t ldo2;
  int N1;
  int interleaved;       // act 3 to 5: gate and up rows alternate in blocks of eight, else gate rows before up rows
  int act_from;          // act 1: rows from this one on
  int x_f32;
  float limit, alpha;    // act 5
  const void* mul;       // act 6: T [mul_rows, ldm]
  const int64_t* ids;    // ... and its rows, [M]
  int64_t ldm, mul_rows;
};

__host__ __device__ __forceinline__ bool gated(int act) { return act >= 3 && act <= 5; }

// clamped gated unit
__device__ __forceinline__ float clamped_unit(float g, float u, float limit, float alpha) {
  g = fminf(g, limit);
  return g / (1.0f + expf(-alpha * g)) * (fminf(fmaxf(u, -limit), limit) + 1.0f);
}

template <typename T>
__device__ __forceinline__ const T* weight_row(const GemvRowsArgs& a, int n) {
  return n < a.N1 ? reinterpret_cast<const T*>(a.w) + (int64_t)n * a.ldw
                  : reinterpret_cast<const T*>(a.w2) + (int64_t)(n - a.N1) * a.ldw;
}

template <typename T>
__device__ __forceinline__ float bias_of(const GemvRowsArgs& a, int n) {
  return a.bias != nullptr ? DT<T>::to_f(reinterpret_cast<const T*>(a.bias)[n]) : 0.f;
}

// hidden unit i of token m from its two products (weight rows ng and nu)
template <typename T>
__device__ __forceinline__ void store_gated(const GemvRowsArgs& a, int m, int i, int ng, int nu, float g, float u) {
  const float z = g + bias_of<T>(a, ng);
  u += bias_of<T>(a, nu);
  const float v = a.act == 5 ? clamped_unit(z, u, a.limit, a.alpha) : (a.act == 4 ? silu(z) : gelu_tanh(z)) * u;
  reinterpret_cast<T*>(a.out)[(int64_t)m * a.ldo + i] = DT<T>::from_f(v);
}

template <typename T>
__device__ __forceinline__ void store_row(const GemvRowsArgs& a, int m, int n, float v) {
  if (n >= a.N1) {
    a.out2[(int64_t)m * a.ldo2 + n - a.N1] = v;
    return;
  }
  v += bias_of<T>(a, n);
  if (a.act == 1 && n >= a.act_from) {
    v = v > 0.f ? v * v : 0.f;
  } else if (a.act == 6) {
    const int64_t row = min(max(a.ids[m], (int64_t)0), a.mul_rows - 1);
    v = gelu_tanh(v) * DT<T>::to_f(reinterpret_cast<const T*>(a.mul)[row * a.ldm + n]);
  }
  if (a.out_mode == 0) {
    reinterpret_cast<T*>(a.out)[(int64_t)m * a.ldo + n] = DT<T>::from_f(v);
  } else {
    float* o = reinterpret_cast<float*>(a.out) + (int64_t)m * a.ldo + n;
    if (a.out_mode == 1) *o += v;
    else *o = a.softcap > 0.f ? a.softcap * tanhf(v / a.softcap) : v;
  }
}

// GLU: a task is a hidden unit, its two rows are the gate's and the up product's.
template <typename T, int M, int R, bool GLU>
__global__ void __launch_bounds__(kThreads) gemv_rows_kernel(GemvRowsArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[kWarps];
  T* sx = reinterpret_cast<T*>(smem);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ntask = (a.N + R - 1) / R;
  const int t0 = blockIdx.x * kWarps + warp;
  auto row_of = [&](int t, int r) {
    if constexpr (GLU) return a.interleaved ? (t >> 3) * 16 + (t & 7) + 8 * r : t + r * (a.N / 2);
    else return t * R + r;
  };
  pdl_launch_dependents();
  if (a.vec && t0 < ntask && lane < R && row_of(t0, lane) < a.N)
    prefetch_l2_bulk(weight_row<T>(a, row_of(t0, lane)), (uint32_t)(a.K * sizeof(T)));
  pdl_wait();
  stage_rows<T>(sx, a.kp, a.x, a.ldx, reinterpret_cast<const T*>(a.norm_w), a.eps, a.M, a.K, red, a.x_f32 != 0);
  for (int t = t0; t < ntask; t += gridDim.x * kWarps) {
    const T* w[R];
#pragma unroll
    for (int r = 0; r < R; ++r) w[r] = weight_row<T>(a, min(row_of(t, r), a.N - 1));
    float acc[M][R] = {};
    dot_rows<T, M, R>(w, sx, a.kp, a.K, a.vec != 0, lane, acc);
    if constexpr (GLU) {
#pragma unroll
      for (int m = 0; m < M; ++m)
        if (lane == m && m < a.M) store_gated<T>(a, m, t, row_of(t, 0), row_of(t, 1), acc[m][0], acc[m][1]);
      continue;
    }
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int n = t * R + r;
        if (lane == ((m * R + r) & 31) && m < a.M && n < a.N) {
          store_row<T>(a, m, n, acc[m][r]);
        }
      }
  }
}

template <typename T>
__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
  else
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// eight fp32 values in T
template <typename T>
__device__ __forceinline__ uint4 converted(const float* p) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  __align__(16) T o[8] = {DT<T>::from_f(a.x), DT<T>::from_f(a.y), DT<T>::from_f(a.z), DT<T>::from_f(a.w),
                          DT<T>::from_f(b.x), DT<T>::from_f(b.y), DT<T>::from_f(b.z), DT<T>::from_f(b.w)};
  return *reinterpret_cast<const uint4*>(o);
}

// 16-bit weights on the tensor cores, NT * 8 tokens: a tile is 16 weight rows (the A operand, straight from global
// memory), `split` warps of the CTA share its K range and meet once per tile in shared memory.  The k order inside a
// 32-wide block is permuted alike for both operands, so that a lane's fragment is one 16-byte load: lane (g, t) holds
// k = 8 t .. 8 t + 7 of rows g and g + 8, and of token g.  Normed rows are staged in shared memory; plain
// activations are read where they are (a CTA reads each value about once).
template <typename T, int NT>
__global__ void __launch_bounds__(kThreads) gemv_mma_kernel(GemvRowsArgs a, int split) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[kWarps];
  constexpr int U = NT == 1 ? 4 : 2;
  float* part = reinterpret_cast<float*>(smem);                         // [2][kWarps][NT * 128]
  T* sx = reinterpret_cast<T*>(smem + 2 * kWarps * NT * 128 * sizeof(float));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int tpc = kWarps / split, sub = warp % split;
  const int ntile = (a.N + 15) / 16, nkb = (a.K + 31) / 32;
  const int per = (nkb + split - 1) / split, kb0 = sub * per, kb1 = min(kb0 + per, nkb);
  pdl_launch_dependents();
  {
    const int tile = blockIdx.x * tpc + warp / split, row = tile * 16 + lane;
    const int k0 = kb0 * 32, bytes = (min(kb1 * 32, a.K) - k0) * (int)sizeof(T);
    if (lane < 16 && row < a.N && bytes > 0) prefetch_l2_bulk(weight_row<T>(a, row) + k0, (uint32_t)bytes);
  }
  pdl_wait();
  const bool staged = a.norm_w != nullptr;
  if (staged)
    stage_rows<T>(sx, a.kp, a.x, a.ldx, reinterpret_cast<const T*>(a.norm_w), a.eps, a.M, a.K, red);
  const T* xs[NT];
  const float* xf[NT];           // rows of the 32-bit stream, converted on the way
  bool xon[NT];
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const int m = n * 8 + g;
    xon[n] = m < a.M;
    xs[n] = (staged ? sx + (size_t)(xon[n] ? m : 0) * a.kp
                    : reinterpret_cast<const T*>(a.x) + (int64_t)(xon[n] ? m : 0) * a.ldx) + t * 8;
    xf[n] = reinterpret_cast<const float*>(a.x) + (int64_t)(xon[n] ? m : 0) * a.ldx + t * 8;
  }
  int par = 0;
  for (int base = blockIdx.x * tpc; base < ntile; base += gridDim.x * tpc, par ^= 1) {
    const int tile = base + warp / split;
    float acc[2][NT][4] = {};
    if (tile < ntile) {
      const T* w0 = weight_row<T>(a, min(tile * 16 + g, a.N - 1)) + t * 8;
      const T* w1 = weight_row<T>(a, min(tile * 16 + g + 8, a.N - 1)) + t * 8;
      for (int kb = kb0; kb < kb1; kb += U) {
        uint4 r0[U], r1[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int k = (kb + u) * 32;
          const bool in = kb + u < kb1 && k + t * 8 < a.K;
          r0[u] = in ? ldg_nc_v4(w0 + k) : make_uint4(0, 0, 0, 0);
          r1[u] = in ? ldg_nc_v4(w1 + k) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int k = (kb + u) * 32;
          const bool in = kb + u < kb1 && k + t * 8 < a.K;
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            uint4 x = make_uint4(0, 0, 0, 0);
            if (in && xon[n]) x = a.x_f32 ? converted<T>(xf[n] + k) : *reinterpret_cast<const uint4*>(xs[n] + k);
            mma16816<T>(acc[0][n], r0[u].x, r1[u].x, r0[u].y, r1[u].y, x.x, x.y);
            mma16816<T>(acc[1][n], r0[u].z, r1[u].z, r0[u].w, r1[u].w, x.z, x.w);
          }
        }
      }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[0][n][i] += acc[1][n][i];
    // accumulator i of lane (g, t): weight row g + 8 * (i / 2), token n * 8 + 2 t + (i & 1)
    if (split > 1) {
      float* mine = part + ((size_t)par * kWarps + warp) * (NT * 128);
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) mine[(n * 4 + i) * 32 + lane] = acc[0][n][i];
      __syncthreads();
      // the group's warps share the sums: value (n, i) goes to warp (n * 4 + i) % split
      const float* grp = part + ((size_t)par * kWarps + warp / split * split) * (NT * 128);
      if (gated(a.act)) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int i = 0; i < 2; ++i)
            if ((n * 2 + i) % split == sub) {
              float gv = 0.f, uv = 0.f;
              for (int w = 0; w < split; ++w) {
                gv += grp[w * (NT * 128) + (n * 4 + i) * 32 + lane];
                uv += grp[w * (NT * 128) + (n * 4 + i + 2) * 32 + lane];
              }
              const int row = tile * 16 + g, m = n * 8 + 2 * t + i;
              if (tile < ntile && m < a.M) store_gated<T>(a, m, tile * 8 + g, row, row + 8, gv, uv);
            }
        continue;
      }
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if ((n * 4 + i) % split == sub) {
            float v = 0.f;
            for (int w = 0; w < split; ++w) v += grp[w * (NT * 128) + (n * 4 + i) * 32 + lane];
            const int row = tile * 16 + g + 8 * (i >> 1), m = n * 8 + 2 * t + (i & 1);
            if (tile < ntile && row < a.N && m < a.M) store_row<T>(a, m, row, v);
          }
    } else if (gated(a.act)) {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int row = tile * 16 + g, m = n * 8 + 2 * t + i;
          if (tile < ntile && m < a.M)
            store_gated<T>(a, m, tile * 8 + g, row, row + 8, acc[0][n][i], acc[0][n][i + 2]);
        }
    } else {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int row = tile * 16 + g + 8 * (i >> 1), m = n * 8 + 2 * t + (i & 1);
          if (tile < ntile && row < a.N && m < a.M) store_row<T>(a, m, row, acc[0][n][i]);
        }
    }
  }
}

int sm_count() {
  static int sms = [] {
    int dev = 0, n = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
    return n;
  }();
  return sms;
}

template <typename T, int M, int R, bool GLU = false>
cudaError_t launch_gemv(GemvRowsArgs& a, bool pdl, cudaStream_t st) {
  auto kern = gemv_rows_kernel<T, M, R, GLU>;
  const size_t smem = (size_t)M * a.kp * sizeof(T);      // rows past a.M are read (and dropped), never used
  if (smem > 40 * 1024) {                 // (static shared memory counts against the default limit too)
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  const int ntask = (a.N + R - 1) / R;
  const int per_sm = smem > 100 * 1024 ? 1 : 2;
  const int want = (ntask + kWarps - 1) / kWarps, cap = sm_count() * per_sm;
  return launch_kernel(kern, dim3(want < cap ? want : cap), dim3(kThreads), smem, st, pdl, a);
}

template <typename T, int M>
cudaError_t pick_rows(GemvRowsArgs& a, bool pdl, cudaStream_t st) {
  const int warps = sm_count() * kWarps;
  if (gated(a.act)) return launch_gemv<T, M, 2, true>(a, pdl, st);
  if (a.N >= 4 * warps) return launch_gemv<T, M, 4>(a, pdl, st);
  if (a.N >= warps) return launch_gemv<T, M, 2>(a, pdl, st);
  return launch_gemv<T, M, 1>(a, pdl, st);
}

template <typename T, int NT>
cudaError_t launch_gemv_mma(GemvRowsArgs& a, bool pdl, cudaStream_t st) {
  auto kern = gemv_mma_kernel<T, NT>;
  a.kp = (a.K + 31) / 32 * 32 + 32;        // 64 bytes of skew between rows: neighbouring tokens in different banks
  const size_t smem = (size_t)2 * kWarps * NT * 128 * sizeof(float) + (a.norm_w != nullptr ? (size_t)a.M * a.kp * sizeof(T) : 0);
  if (smem > 226 * 1024) return cudaErrorInvalidValue;
  if (smem > 40 * 1024) {                 // (static shared memory counts against the default limit too)
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  // enough warps for the machine, at least four k blocks each
  const int ntile = (a.N + 15) / 16, nkb = (a.K + 31) / 32, want = sm_count() * 2 * kWarps;
  int split = 1;
  while (split < kWarps && ntile * split < want && nkb / (2 * split) >= 4) split *= 2;
  const int tpc = kWarps / split, ctas = (ntile + tpc - 1) / tpc, cap = sm_count() * 2;
  return launch_kernel(kern, dim3(ctas < cap ? ctas : cap), dim3(kThreads), smem, st, pdl, a, split);
}

int g_mma_from = 1;      // smallest row count that takes the tensor-core kernel
bool mma_from(const GemvRowsArgs& a) { return a.M >= g_mma_from; }

template <typename T>
cudaError_t pick_m(GemvRowsArgs& a, bool pdl, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    const bool direct = a.norm_w != nullptr || ((reinterpret_cast<uintptr_t>(a.x) & 15) == 0 && a.ldx % (a.x_f32 ? 4 : 8) == 0);
    if (a.vec && direct && mma_from(a) && (!gated(a.act) || a.interleaved)) {
      if (a.M <= 8) return launch_gemv_mma<T, 1>(a, pdl, st);
      return launch_gemv_mma<T, 2>(a, pdl, st);
    }
  }
  if (a.M > 8) return cudaErrorInvalidValue;
  if (a.M == 1) return pick_rows<T, 1>(a, pdl, st);
  if (a.M == 2) return pick_rows<T, 2>(a, pdl, st);
  if (a.M <= 4) return pick_rows<T, 4>(a, pdl, st);
  return pick_rows<T, 8>(a, pdl, st);
}

// ------------------------------------------------------------------------------------------------ mixture of experts
struct RouterArgs {
  const float* x;        // residual stream [tokens, K]
  const void* norm_w;
  const void* w;         // [E, K]
  float* weights;        // [tokens, k]
  int64_t* idx;          // [tokens, k]
  int64_t ldx;
  float eps;
  int K, E, k;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) moe_router_kernel(RouterArgs a) {
  extern __shared__ __align__(16) float sh[];      // [K] normed row, [E] scores
  __shared__ float red[kWarps];
  float* h = sh;
  float* sc = sh + a.K;
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const float* src = a.x + (int64_t)t * a.ldx;
  float s = 0.f;
  for (int k = threadIdx.x; k < a.K; k += kThreads) {
    const float v = src[k];
    h[k] = v;
    s = fmaf(v, v, s);
  }
  s = block_sum(s, red);
  const float inv = 1.0f / sqrtf(s / (float)a.K + a.eps);
  const T* nw = reinterpret_cast<const T*>(a.norm_w);
  for (int k = threadIdx.x; k < a.K; k += kThreads) h[k] *= inv * DT<T>::to_f(nw[k]);
  __syncthreads();
  for (int e = warp; e < a.E; e += kWarps) {
    const T* w = reinterpret_cast<const T*>(a.w) + (int64_t)e * a.K;
    float acc = 0.f;
    constexpr int VN = Vec<T>::n;
    if (a.K % VN == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0) {
#pragma unroll 4
      for (int v = lane; v < a.K / VN; v += 32) {
        float wf[VN];
        unpack<T>(ldg_nc_v4(reinterpret_cast<const uint4*>(w) + v), wf);
#pragma unroll
        for (int i = 0; i < VN; ++i) acc = fmaf(h[v * VN + i], wf[i], acc);
      }
    } else {
      for (int k = lane; k < a.K; k += 32) acc = fmaf(h[k], DT<T>::to_f(w[k]), acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) sc[e] = 1.0f / (1.0f + expf(-acc));
  }
  __syncthreads();
  if (warp == 0) {
    for (int r = 0; r < a.k; ++r) {
      float best = -1.f;
      int bi = 0x7fffffff;
      for (int e = lane; e < a.E; e += 32)
        if (sc[e] > best) { best = sc[e]; bi = e; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
      }
      if (bi >= a.E) { bi = 0; best = 0.f; }       // scores that are not numbers
      if (lane == 0) {
        a.weights[(int64_t)t * a.k + r] = best;
        a.idx[(int64_t)t * a.k + r] = bi;
        sc[bi] = -2.f;
      }
      __syncwarp();
    }
  }
}

struct SoftRouterArgs {
  const void* h;         // T [tokens, ldh], normed
  const void* w;         // T [E (+ 1), K]: the last row gates a shared expert
  float* weights;        // [tokens, k (+ 1)]
  int64_t* idx;          // [tokens, k (+ 1)]; the shared expert is number E
  int64_t ldh;
  float scale;
  int K, E, k, groups, keep, shared, vec, kp;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) moe_soft_router_kernel(SoftRouterArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[kWarps];
  T* sx = reinterpret_cast<T*>(smem);
  float* sc = reinterpret_cast<float*>(smem + (size_t)a.kp * sizeof(T));     // [E + 1] scores, [groups]
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rows = a.E + a.shared;
  pdl_launch_dependents();
  if (a.vec && warp < rows && lane == 0)
    prefetch_l2_bulk(reinterpret_cast<const T*>(a.w) + (int64_t)warp * a.K, (uint32_t)(a.K * sizeof(T)));
  pdl_wait();
  stage_rows<T>(sx, a.kp, reinterpret_cast<const T*>(a.h) + (int64_t)t * a.ldh, 0, (const T*)nullptr, 0.f, 1, a.K, red);
  for (int e = warp; e < rows; e += kWarps) {
    const T* w[1] = {reinterpret_cast<const T*>(a.w) + (int64_t)e * a.K};
    float acc[1][1] = {};
    dot_rows<T, 1, 1>(w, sx, a.kp, a.K, a.vec != 0, lane, acc);
    if (lane == 0) sc[e] = acc[0][0];
  }
  __syncthreads();
  if (warp != 0) return;
  const int kt = a.k + a.shared;
  if (a.shared && lane == 0) {
    a.weights[(int64_t)t * kt + a.k] = 1.0f / (1.0f + expf(-sc[a.E]));
    a.idx[(int64_t)t * kt + a.k] = a.E;
  }
  softmax_grouped_topk(sc, sc + rows, a.E, a.groups, a.keep, a.k, a.scale, a.weights + (int64_t)t * kt,
                       a.idx + (int64_t)t * kt, lane);
}

struct MoeArgs {
  const void* x;           // glu: residual stream [tokens, K] (normed on the way), or finished rows of T (norm_w null)
  const void* norm_w;
  const void* w;           // glu: [E, 2I, K]; down: [E, N, I]
  const void* y_in;        // down: [tokens * k, ldy]
  void* out;               // glu: T [tokens * k, ldy]; down: fp32 [tokens, N], accumulated into or written
  const float* weights;    // [tokens, k]
  const int64_t* idx;      // [tokens, k]
  int64_t ldx, ldo;
  float eps, limit, alpha;
  int K, I, E, k, kp;
  int tile;                // gate / up rows in alternating tiles of this many rows; 0: gate rows then up rows
  int vec;
  int act;                 // glu: 2 clamped, on weighted inputs; 4 silu(gate) * up; 5 clamped
  const void* ws;          // the shared expert, number E of idx: glu [2 Is, K], down [N, Is]
  int Is, vec_s, tile_s;
  int64_t ldy;             // row stride of the hidden units (at least I and Is)
  int weighted;            // down: weights applied here
  int add;                 // down: results added instead of written
  float limit_s;           // clamp of the shared expert
};

template <typename T>
__global__ void __launch_bounds__(kThreads) moe_glu_kernel(MoeArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[kWarps];
  T* sx = reinterpret_cast<T*>(smem);
  const int slot = blockIdx.y, t = slot / a.k;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int e = (int)a.idx[slot];
  const bool shared = e == a.E;
  const int64_t row = (int64_t)t * a.ldx;
  stage_rows<T>(sx, a.kp, a.norm_w != nullptr ? (const void*)(reinterpret_cast<const float*>(a.x) + row)
                                              : (const void*)(reinterpret_cast<const T*>(a.x) + row),
                0, reinterpret_cast<const T*>(a.norm_w), a.eps, 1, a.K, red);
  const T* W = shared ? reinterpret_cast<const T*>(a.ws) : reinterpret_cast<const T*>(a.w) + (int64_t)e * 2 * a.I * a.K;
  const int I = shared ? a.Is : a.I, tile = shared ? a.tile_s : a.tile;
  const bool vec = shared ? a.vec_s != 0 : a.vec != 0;
  const float rw = a.weights[slot];
  for (int i = blockIdx.x * kWarps + warp; i < I; i += gridDim.x * kWarps) {
    const int g = tile > 0 ? i / tile * 2 * tile + i % tile : i;
    const int u = tile > 0 ? g + tile : I + i;
    const T* w[2] = {W + (int64_t)g * a.K, W + (int64_t)u * a.K};
    float acc[1][2] = {};
    dot_rows<T, 1, 2>(w, sx, a.kp, a.K, vec, lane, acc);
    if (lane == 0) {
      const float y = a.act == 4   ? silu(acc[0][0]) * acc[0][1]
                      : a.act == 5 ? clamped_unit(acc[0][0], acc[0][1], shared ? a.limit_s : a.limit, a.alpha)
                                   : clamped_unit(acc[0][0] * rw, acc[0][1] * rw, a.limit, a.alpha);
      reinterpret_cast<T*>(a.out)[(int64_t)slot * a.ldy + i] = DT<T>::from_f(y);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(kThreads) moe_down_kernel(MoeArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[kWarps];
  T* sx = reinterpret_cast<T*>(smem);
  const int t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const T* y = reinterpret_cast<const T*>(a.y_in) + (int64_t)t * a.k * a.ldy;
  const int own = a.Is > 0 ? a.k - 1 : a.k;            // a shared expert is the last choice
  stage_rows<T>(sx, a.kp, y, a.ldy, (const T*)nullptr, 0.f, own, a.I, red);
  if (own < a.k)
    stage_rows<T>(sx + (size_t)own * a.kp, a.kp, y + own * a.ldy, 0, (const T*)nullptr, 0.f, 1, a.Is, red);
  const int N = a.K;
  for (int n2 = blockIdx.x * kWarps + warp; n2 * 2 < N; n2 += gridDim.x * kWarps) {
    const int n = n2 * 2;
    float s0 = 0.f, s1 = 0.f;
    for (int j = 0; j < a.k; ++j) {
      const bool shared = j >= own;
      const int I = shared ? a.Is : a.I;
      const T* We = shared ? reinterpret_cast<const T*>(a.ws)
                           : reinterpret_cast<const T*>(a.w) + a.idx[(int64_t)t * a.k + j] * (int64_t)N * I;
      const T* w[2] = {We + (int64_t)n * I, We + (int64_t)min(n + 1, N - 1) * I};
      float acc[1][2] = {};
      dot_rows<T, 1, 2>(w, sx + (size_t)j * a.kp, a.kp, I, shared ? a.vec_s != 0 : a.vec != 0, lane, acc);
      const float f = a.weighted ? a.weights[(int64_t)t * a.k + j] : 1.0f;
      s0 = fmaf(f, acc[0][0], s0);
      s1 = fmaf(f, acc[0][1], s1);
    }
    float* o = reinterpret_cast<float*>(a.out) + (int64_t)t * a.ldo + n;
    if (lane == 0) o[0] = a.add ? o[0] + s0 : s0;
    if (lane == 1 && n + 1 < N) o[1] = a.add ? o[1] + s1 : s1;
  }
}

template <typename T>
int padded(int K) { return (K + Vec<T>::n - 1) / Vec<T>::n * Vec<T>::n; }

template <typename T>
int vec_ok(const void* p, int64_t ld, int K) {
  return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && ld % Vec<T>::n == 0 && K % Vec<T>::n == 0;
}

template <typename K>
cudaError_t allow_smem(K kern, size_t smem) {
  if (smem <= 40 * 1024) return cudaSuccess;      // static shared memory counts against the default limit too
  if (smem > 226 * 1024) return cudaErrorInvalidValue;
  return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

}  // namespace

// Rows of x one call may take.  Normed rows are staged in shared memory, which may allow fewer (the call says so).
IPEX_API int ipex_gemv_rows_max(int K, int dtype) {
  if (dtype != DT_F32 && K % 8 == 0) return 16;
  const int64_t row = ((int64_t)K + 8) * (dtype == DT_F32 ? 4 : 2);
  const int64_t m = (200 * 1024) / row;
  return m >= 8 ? 8 : m >= 4 ? 4 : m >= 2 ? 2 : (int)m;
}

// Timing sweeps: smallest row count of the tensor-core kernel (17: never).
IPEX_API void ipex_gemv_rows_tune(int mma_from_rows) { g_mma_from = mma_from_rows; }

// y = act(x . W^T + bias): see GemvRowsArgs.  M <= ipex_gemv_rows_max(K, dtype).  w2 / out2 (may be null): N2 more
// rows with the same row stride whose results go to out2 [M, ldo2] in fp32.  act 1: rows from act_from on.  act 3 to 5:
// out_mode 0, N even (a multiple of 16 when interleaved), no second matrix.  act 6: out_mode 0, `mul` [mul_rows, ldm] and the
// tokens' rows of it, ids [M].  x_f32: x is fp32 and converted (norm_w null).
IPEX_API int ipex_gemv_rows(const void* w, int64_t ldw, const void* x, int64_t ldx, const void* norm_w, float eps,
                            const void* bias, void* out, int64_t ldo, const void* w2, int N2, float* out2, int64_t ldo2,
                            int M, int N, int K, int out_mode, int act, int interleaved, float softcap, int x_f32,
                            int act_from, float limit, float alpha, const void* mul, int64_t ldm, int64_t mul_rows,
                            const int64_t* ids, int dtype, int pdl, void* stream) {
  if (M < 1 || N < 1 || K < 1 || out_mode < 0 || out_mode > 2 || M > ipex_gemv_rows_max(K, dtype))
    return (int)cudaErrorInvalidValue;
  if (act < 0 || act == 2 || act > 6 || (gated(act) && (out_mode != 0 || (N % 2) || (interleaved && (N % 16)) || w2 != nullptr)) ||
      (act == 6 && (out_mode != 0 || mul == nullptr || ids == nullptr || mul_rows < 1)) || (x_f32 && norm_w != nullptr) ||
      (w2 != nullptr && (N2 < 1 || out2 == nullptr)))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    GemvRowsArgs a = {w, x, norm_w, out, ldw, ldx, ldo, eps, softcap, M, N, K, padded<T>(K), out_mode, act, 0};
    a.bias = bias;
    a.N1 = N;
    a.interleaved = interleaved;
    a.x_f32 = x_f32;
    a.act_from = act_from;
    a.limit = limit;
    a.alpha = alpha;
    a.mul = mul;
    a.ids = ids;
    a.ldm = ldm;
    a.mul_rows = mul_rows;
    if (w2 != nullptr) {
      a.w2 = w2;
      a.out2 = out2;
      a.ldo2 = ldo2;
      a.N = N + N2;
    }
    a.vec = vec_ok<T>(w, ldw, K) && (w2 == nullptr || vec_ok<T>(w2, ldw, K));
    return pick_m<T>(a, pdl != 0, (cudaStream_t)stream);
  });
}

// Router of `tokens` rows of the residual stream: weights = the k largest sigmoid scores, idx = their experts
// (descending score, the lower index first among equals).
IPEX_API int ipex_moe_router_sigmoid(const float* x, int64_t ldx, const void* norm_w, float eps, const void* w,
                                     float* weights, int64_t* idx, int tokens, int K, int E, int k, int dtype, int pdl,
                                     void* stream) {
  if (tokens < 1 || K < 1 || E < 1 || k < 1 || k > E) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    RouterArgs a = {x, norm_w, w, weights, idx, ldx, eps, K, E, k};
    const size_t smem = ((size_t)K + E) * sizeof(float);
    cudaError_t e = allow_smem(moe_router_kernel<T>, smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(moe_router_kernel<T>, dim3(tokens), dim3(kThreads), smem, (cudaStream_t)stream, pdl != 0, a);
  });
}

// Router from finished rows h: soft-max over E experts, choice among the `keep` best of `groups` equal groups, weights
// divided by their sum and times scale; shared: row E of w gates a shared expert, which becomes choice k (number E).
IPEX_API int ipex_moe_router_softmax(const void* h, int64_t ldh, const void* w, float* weights, int64_t* idx, int tokens,
                                     int K, int E, int groups, int keep, int k, int shared, float scale, int dtype, int pdl,
                                     void* stream) {
  if (tokens < 1 || K < 1 || E < 1 || k < 1 || groups < 1 || E % groups || keep < 1 || keep > groups || k > E / groups * keep)
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    SoftRouterArgs a = {h, w, weights, idx, ldh, scale, K, E, k, groups, keep, shared != 0, vec_ok<T>(w, K, K), padded<T>(K)};
    const size_t smem = (size_t)a.kp * sizeof(T) + ((size_t)E + 1 + groups) * sizeof(float);
    cudaError_t e = allow_smem(moe_soft_router_kernel<T>, smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(moe_soft_router_kernel<T>, dim3(tokens), dim3(kThreads), smem, (cudaStream_t)stream, pdl != 0, a);
  });
}

// First half of the experts for `tokens` rows.  act 2: y[token * k + j] = g * sigmoid(alpha g) * (u + 1), g = min(gate,
// limit), u = clamp(up, +-limit), gate / up of expert idx[token, j] on weight * norm(x).  act 4: silu(gate) * up of
// finished rows x (norm_w null); act 5: the clamped unit of them, the shared expert's with limit_s.  ws (may be null): the shared expert's rows, [2 Is, K]; tile / tile_s: see MoeArgs.
IPEX_API int ipex_moe_glu_rows(const void* x, int64_t ldx, const void* norm_w, float eps, const void* w, const void* ws,
                               void* y, int64_t ldy, const float* weights, const int64_t* idx, int tokens, int K, int I,
                               int Is, int E, int k, int act, float limit, float limit_s, float alpha, int tile, int tile_s,
                               int dtype, int pdl, void* stream) {
  if (tokens < 1 || K < 1 || I < 1 || k < 1 || (int64_t)tokens * k > 65535 || tile < 0 || (tile > 0 && I % tile != 0) ||
      Is < 0 || (Is > 0 && (ws == nullptr || act == 2)) || tile_s < 0 || (tile_s > 0 && Is % tile_s != 0) || ldy < I ||
      ldy < Is || (act != 2 && act != 4 && act != 5) || (act == 2) != (norm_w != nullptr))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    MoeArgs a = {};
    a.x = x; a.norm_w = norm_w; a.w = w; a.out = y; a.weights = weights; a.idx = idx; a.ldx = ldx; a.eps = eps;
    a.limit = limit; a.limit_s = limit_s; a.alpha = alpha; a.K = K; a.I = I; a.E = E; a.k = k; a.kp = padded<T>(K); a.act = act;
    a.ws = ws; a.Is = Is; a.ldy = ldy; a.tile = tile; a.tile_s = tile_s;
    a.vec = vec_ok<T>(w, K, K);
    a.vec_s = ws != nullptr && vec_ok<T>(ws, K, K);
    const size_t smem = (size_t)a.kp * sizeof(T);
    cudaError_t e = allow_smem(moe_glu_kernel<T>, smem);
    if (e != cudaSuccess) return e;
    const int slots = tokens * k, want = ((I > Is ? I : Is) + kWarps - 1) / kWarps;
    const int cap = (sm_count() * 4 + slots - 1) / slots;
    return launch_kernel(moe_glu_kernel<T>, dim3(want < cap ? want : cap, slots), dim3(kThreads), smem,
                         (cudaStream_t)stream, pdl != 0, a);
  });
}

// Second half: sum_j down_{idx[token, j]}(y[token * k + j]), weighted unless weights is null, added to out or (add 0) written.
// ws (may be null): the shared expert's rows, [N, Is]; it is then the last of the k choices.
IPEX_API int ipex_moe_down_rows(const void* y, int64_t ldy, const void* w, const void* ws, const float* weights, float* out,
                                int64_t ldo, const int64_t* idx, int tokens, int N, int I, int Is, int E, int k, int add,
                                int dtype, int pdl, void* stream) {
  if (tokens < 1 || tokens > 65535 || N < 1 || I < 1 || k < 1 || Is < 0 || (Is > 0 && (ws == nullptr || k < 2)) ||
      ldy < I || ldy < Is)
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    MoeArgs a = {};
    a.y_in = y; a.w = w; a.out = out; a.idx = idx; a.ldo = ldo; a.K = N; a.I = I; a.E = E; a.k = k;
    a.kp = padded<T>(I > Is ? I : Is);
    a.weights = weights; a.weighted = weights != nullptr; a.add = add; a.ws = ws; a.Is = Is; a.ldy = ldy;
    a.vec = vec_ok<T>(w, I, I);
    a.vec_s = ws != nullptr && vec_ok<T>(ws, Is, Is);
    const size_t smem = (size_t)a.kp * k * sizeof(T);
    cudaError_t e = allow_smem(moe_down_kernel<T>, smem);
    if (e != cudaSuccess) return e;
    const int want = (N / 2 + kWarps) / kWarps, cap = (sm_count() * 4 + tokens - 1) / tokens;
    return launch_kernel(moe_down_kernel<T>, dim3(want < cap ? want : cap, tokens), dim3(kThreads), smem,
                         (cudaStream_t)stream, pdl != 0, a);
  });
}
