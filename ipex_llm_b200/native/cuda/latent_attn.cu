// Multi-head latent attention against a cache of latents, sm_100a.
//
// A token's cache row is [ latent c (R values, RMS-normed) | rotated key part shared by all heads (rd values) | zeros ],
// so attention never materialises per-head keys or values.  With the up-projections absorbed into the query and the
// output, the score of head h is  (W_uk[h]^T q_h) . c + q_rot_h . k_rot  and the head's output  W_uv[h] (sum_j p_j c_j):
// multi-query attention over rows of R + rd values.  Three kernels per layer and step:
//
//   latent_prep     q_abs = W_uk[h]^T q_h for every head, rotation of the query parts in place, and the new tokens'
//                   latent (norm) and key part (rotation) appended to the cache
//   latent_attn     split over the visible keys (sliding window / all), online soft-max, partial sums to scratch
//   latent_uv       merge of the splits and the value up-projection, [tokens, H * vd]
//
// Every query token is described by (cache row `slot`, position `pos`); `start[slot]` is the position of the sequence's
// first token.  Tokens of different sequences and lengths share a launch; a prompt portion is simply many query tokens.
// `latent_prompt_prep` is the first kernel of the prompt path, whose attention runs on expanded keys and values
// (latent_prefill_tcgen05.cu).
//
// The 16-bit attention kernel feeds mma.sync from one shared-memory tile of cache rows that serves as keys and as
// values for up to 32 heads: decode is bound by the cache rows it streams, not by the tensor rate.  The generic kernel
// takes every size and 32-bit models.
#include "common/utils.cuh"

namespace {

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

template <typename T> struct Vec {
  static constexpr int n = 16 / sizeof(T);
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
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

struct PrepArgs {
  void* q;              // T [M, ldq]: per head [dim | rd]
  const void* kv;       // T [M, ldkv]: R latents, then rd key values; null: the cache holds the tokens' rows already
  const void* norm_w;   // T [R]
  const void* w_uk;     // T [H * dim, R]
  const float* cosp;    // [positions, half]
  const float* sinp;
  const int* slot;      // [M]
  const int* pos;       // [M]
  const int* start;     // [slots]
  void* cache;          // T, row (slot, position) at slot * slot_stride + position * ldc
  void* qabs;           // T [M, H, R]
  void* c_out;          // prompt path: T [M, ld_c]
  void* kr_out;         // prompt path: T [M, ld_kr]
  int64_t ldq, ldkv, slot_stride, ldc, ld_c, ld_kr;
  float eps;
  int M, H, dim, rd, R, half;
};

// rotate pairs (i, i + half) of one vector in place: threads of the block share the work
template <typename T>
__device__ __forceinline__ void rotate_pair(T* v, int i, int half, float c, float s) {
  const float a = DT<T>::to_f(v[i]), b = DT<T>::to_f(v[i + half]);
  v[i] = DT<T>::from_f(a * c - b * s);
  v[i + half] = DT<T>::from_f(b * c + a * s);
}

// norm of the latent part, rotation of the key part, append to the cache (whole block, one token)
template <typename T>
__device__ void append_token(const PrepArgs& a, int m, float* red) {
  const T* row = reinterpret_cast<const T*>(a.kv) + (int64_t)m * a.ldkv;
  const T* nw = reinterpret_cast<const T*>(a.norm_w);
  const int s = a.slot[m], p = a.pos[m], rel = p - a.start[s];
  T* dst = reinterpret_cast<T*>(a.cache) + (int64_t)s * a.slot_stride + (int64_t)p * a.ldc;
  float ss = 0.f;
  for (int r = threadIdx.x; r < a.R; r += blockDim.x) {
    const float v = DT<T>::to_f(row[r]);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)a.R + a.eps);
  for (int r = threadIdx.x; r < a.R; r += blockDim.x) {
    const T v = DT<T>::from_f(DT<T>::to_f(row[r]) * inv * DT<T>::to_f(nw[r]));
    dst[r] = v;
    if (a.c_out != nullptr) reinterpret_cast<T*>(a.c_out)[(int64_t)m * a.ld_c + r] = v;
  }
  const float* cp = a.cosp + (int64_t)rel * a.half;
  const float* sp = a.sinp + (int64_t)rel * a.half;
  for (int i = threadIdx.x; i < a.rd; i += blockDim.x) {
    float v = DT<T>::to_f(row[a.R + i]);
    if (i < a.half) v = v * cp[i] - DT<T>::to_f(row[a.R + i + a.half]) * sp[i];
    else if (i < 2 * a.half) v = v * cp[i - a.half] + DT<T>::to_f(row[a.R + i - a.half]) * sp[i - a.half];
    const T o = DT<T>::from_f(v);
    dst[a.R + i] = o;
    if (a.kr_out != nullptr) reinterpret_cast<T*>(a.kr_out)[(int64_t)m * a.ld_kr + i] = o;
  }
}

constexpr int kPrepThreads = 256;
constexpr int kPrepCols = 128;     // latent columns per block

// grid (H * column blocks + 1, token groups of MT): the last x block appends the group's tokens to the cache (and is not
// launched when there is nothing to append).
template <typename T, int V, int MT>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(PrepArgs a) {
  __shared__ float red[kPrepThreads / 32];
  constexpr int TC = kPrepCols / V;           // threads along the columns
  constexpr int DG = kPrepThreads / TC;       // groups along the head dimension
  __shared__ float part[DG][kPrepCols + 1];
  extern __shared__ float sq[];               // [MT][dim]
  const int cb = (a.R + kPrepCols - 1) / kPrepCols;
  const int m0 = blockIdx.y * MT, mn = min(MT, a.M - m0);
  pdl_launch_dependents();
  pdl_wait();
  if ((int)blockIdx.x == a.H * cb) {
    for (int m = 0; m < mn; ++m) append_token<T>(a, m0 + m, red);
    return;
  }
  const int h = blockIdx.x / cb, c0 = (blockIdx.x % cb) * kPrepCols;
  T* q0 = reinterpret_cast<T*>(a.q) + (int64_t)m0 * a.ldq + (int64_t)h * (a.dim + a.rd);
  if (c0 == 0) {
    for (int i = threadIdx.x; i < mn * a.half; i += kPrepThreads) {
      const int m = i / a.half, j = i % a.half;
      const int64_t rel = a.pos[m0 + m] - a.start[a.slot[m0 + m]];
      rotate_pair<T>(q0 + (int64_t)m * a.ldq + a.dim, j, a.half, a.cosp[rel * a.half + j], a.sinp[rel * a.half + j]);
    }
  }
  for (int i = threadIdx.x; i < MT * a.dim; i += kPrepThreads) {
    const int m = i / a.dim, d = i % a.dim;
    sq[i] = m < mn ? DT<T>::to_f(q0[(int64_t)m * a.ldq + d]) : 0.f;
  }
  __syncthreads();
  const int tc = threadIdx.x % TC, dg = threadIdx.x / TC;
  const int col = c0 + tc * V;
  float acc[MT][V] = {};
  if (col < a.R) {
    const T* w = reinterpret_cast<const T*>(a.w_uk) + (int64_t)h * a.dim * a.R + col;
#pragma unroll 4
    for (int d = dg; d < a.dim; d += DG) {
      float wf[V];
      if constexpr (V > 1) {
        const uint4 raw = ldg_nc_v4(w + (int64_t)d * a.R);
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < V; ++i) wf[i] = DT<T>::to_f(e[i]);
      } else {
        wf[0] = DT<T>::to_f(w[(int64_t)d * a.R]);
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float qv = sq[m * a.dim + d];
#pragma unroll
        for (int i = 0; i < V; ++i) acc[m][i] = fmaf(qv, wf[i], acc[m][i]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    if (m < mn) {
#pragma unroll
      for (int i = 0; i < V; ++i) part[dg][tc * V + i] = acc[m][i];
      __syncthreads();
      if (threadIdx.x < kPrepCols && c0 + (int)threadIdx.x < a.R) {
        float s = 0.f;
#pragma unroll
        for (int g = 0; g < DG; ++g) s += part[g][threadIdx.x];
        reinterpret_cast<T*>(a.qabs)[((int64_t)(m0 + m) * a.H + h) * a.R + c0 + threadIdx.x] = DT<T>::from_f(s);
      }
      __syncthreads();
    }
  }
}

// one CTA per token: rotation of all heads' query parts in place, cache append, and contiguous copies of the latent
// and key parts for the prompt attention
template <typename T>
__global__ void __launch_bounds__(256) latent_prompt_prep_kernel(PrepArgs a) {
  __shared__ float red[8];
  const int m = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  T* q = reinterpret_cast<T*>(a.q) + (int64_t)m * a.ldq;
  const int64_t rel = a.pos[m] - a.start[a.slot[m]];
  for (int i = threadIdx.x; i < a.H * a.half; i += blockDim.x) {
    const int h = i / a.half, j = i % a.half;
    rotate_pair<T>(q + (int64_t)h * (a.dim + a.rd) + a.dim, j, a.half, a.cosp[rel * a.half + j],
                   a.sinp[rel * a.half + j]);
  }
  if (a.kv != nullptr) append_token<T>(a, m, red);
}

struct LatentAttnArgs {
  const void* qabs;     // T [M, H, R]
  const void* qkv;      // T [M, ldq]; rotated query part of head h at h * (dim + rd) + dim
  const void* cache;
  const int* slot;
  const int* pos;
  const int* start;
  float* o;             // [M, nsplit, H, R] unnormalised partial outputs
  float* ml;            // [M, nsplit, H, 2] running maximum (log2 domain) and sum
  int64_t ldq, slot_stride, ldc;
  float scale_log2;
  int M, H, dim, rd, R, window, nsplit;
};

__device__ __forceinline__ void visible_range(const LatentAttnArgs& a, int m, int split, int align, int& lo, int& hi) {
  const int s = a.slot[m], p = a.pos[m];
  int first = a.start[s];
  if (a.window > 0) first = max(first, p - a.window + 1);
  const int len = p - first + 1;
  const int chunk = ((len + a.nsplit - 1) / a.nsplit + align - 1) / align * align;
  lo = first + split * chunk;
  hi = min(lo + chunk, p + 1);
}

// ------------------------------------------------------------------------------------------------ generic kernel
constexpr int kGenWarps = 4;
template <typename T>
__global__ void __launch_bounds__(kGenWarps * 32) latent_attn_generic_kernel(LatentAttnArgs a) {
  extern __shared__ float sh[];            // q [R + rd], per-warp output [kGenWarps][R]
  __shared__ float sm[kGenWarps], sl[kGenWarps];
  const int h = blockIdx.x, split = blockIdx.y, m = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int D = a.R + a.rd;
  float* q = sh;
  float* acc = sh + D + warp * a.R;
  pdl_launch_dependents();
  pdl_wait();
  const T* qa = reinterpret_cast<const T*>(a.qabs) + ((int64_t)m * a.H + h) * a.R;
  const T* qr = reinterpret_cast<const T*>(a.qkv) + (int64_t)m * a.ldq + (int64_t)h * (a.dim + a.rd) + a.dim;
  for (int i = threadIdx.x; i < D; i += blockDim.x) q[i] = i < a.R ? DT<T>::to_f(qa[i]) : DT<T>::to_f(qr[i - a.R]);
  for (int r = lane; r < a.R; r += 32) acc[r] = 0.f;
  __syncthreads();
  int lo, hi;
  visible_range(a, m, split, 1, lo, hi);
  const T* base = reinterpret_cast<const T*>(a.cache) + (int64_t)a.slot[m] * a.slot_stride;
  float mx = -INFINITY, l = 0.f;
  for (int j = lo + warp; j < hi; j += kGenWarps) {
    const T* row = base + (int64_t)j * a.ldc;
    float s = 0.f;
    for (int i = lane; i < D; i += 32) s = fmaf(q[i], DT<T>::to_f(row[i]), s);
    s = warp_sum(s) * a.scale_log2;
    const float mn = fmaxf(mx, s);
    const float corr = exp2f(mx - mn), p = exp2f(s - mn);
    l = l * corr + p;
    mx = mn;
    for (int r = lane; r < a.R; r += 32) acc[r] = fmaf(p, DT<T>::to_f(row[r]), acc[r] * corr);
  }
  if (lane == 0) { sm[warp] = mx; sl[warp] = l; }
  __syncthreads();
  float M = -INFINITY, L = 0.f, w[kGenWarps];
#pragma unroll
  for (int i = 0; i < kGenWarps; ++i) M = fmaxf(M, sm[i]);
#pragma unroll
  for (int i = 0; i < kGenWarps; ++i) {
    w[i] = sm[i] == -INFINITY ? 0.f : exp2f(sm[i] - M);
    L += w[i] * sl[i];
  }
  const int64_t part = ((int64_t)m * a.nsplit + split) * a.H + h;
  for (int r = threadIdx.x; r < a.R; r += blockDim.x) {
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < kGenWarps; ++i) o += w[i] * sh[D + i * a.R + r];
    a.o[part * a.R + r] = o;
  }
  if (threadIdx.x == 0) { a.ml[part * 2] = M; a.ml[part * 2 + 1] = L; }
}

// ------------------------------------------------------------------------------------------------ tensor-core kernel
constexpr int kKT = 32;         // cache rows per tile
constexpr int kStages = 3;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)) : "memory");
}
template <typename T>
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  else
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// MG groups of 16 heads per CTA, eight warps each.
//   scores  a warp owns a quarter of the row (k) for 16 of the tile's 32 keys; its part of the queries stays in
//           registers for the whole loop, the four partial sums of a score meet in shared memory
//   values  a warp owns RT 8-column tiles of the output for all heads of the CTA
// KS: 16-wide k steps a warp holds (row <= 64 * KS values).
template <typename T, int MG, int RT, int KS>
__global__ void __launch_bounds__(MG * 256) latent_attn_mma_kernel(LatentAttnArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int kHeads = MG * 16, kWarpsHere = MG * 8;
  constexpr int kLdS = kKT + 4;
  const int Dp = (int)a.ldc;                    // R + rd rounded up to a multiple of 64, zero-filled
  const int ld = Dp + 8;                        // shared-memory row: 16 bytes of skew between rows
  T* sK = reinterpret_cast<T*>(smem);           // [kStages][kKT][ld]
  T* sP = sK + kStages * kKT * ld;              // [kHeads][kKT + 8]
  float* sS = reinterpret_cast<float*>(sP + kHeads * (kKT + 8));   // [4][kHeads][kLdS]
  float* sC = sS + 4 * kHeads * kLdS;           // [kHeads] rescale factors
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int mg = warp >> 3, kq = warp & 3, kh = (warp >> 2) & 1;
  static_assert(kHeads <= kKT, "the queries pass through one stage");
  const int h0 = blockIdx.x * kHeads, split = blockIdx.y, m = blockIdx.z;
  pdl_launch_dependents();
  pdl_wait();
  int lo, hi;
  visible_range(a, m, split, kKT, lo, hi);
  const int ntile = hi > lo ? (hi - lo + kKT - 1) / kKT : 0;
  const T* base = reinterpret_cast<const T*>(a.cache) + (int64_t)a.slot[m] * a.slot_stride;
  const int vec_row = Dp / 8;
  auto load_tile = [&](int i) {
    T* dst = sK + (i % kStages) * kKT * ld;
    for (int r = warp; r < kKT; r += kWarpsHere) {
      const T* src = base + (int64_t)min(lo + i * kKT + r, hi - 1) * a.ldc;   // past the end: the last row, masked below
      for (int v = lane; v < vec_row; v += 32) cp_async16(dst + r * ld + v * 8, src + v * 8);
    }
  };
  for (int i = 0; i < kStages - 1; ++i) {
    if (i < ntile) load_tile(i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  // queries [absorbed | rotated | zeros] (heads past H are zero) pass through the stage that the prologue left free
  // into the warp's fragments
  const int ks = Dp / 64, k0 = kq * (Dp / 4);
  const int ar = lane & 15, ac = (lane >> 4) * 8;                   // ldmatrix address of an A fragment
  T* sQ = sK + (kStages - 1) * kKT * ld;
  for (int r = warp; r < kHeads; r += kWarpsHere) {
    const int h = h0 + r;
    const bool on = h < a.H;
    const uint4* qv = reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(a.qabs) +
                                                     ((int64_t)m * a.H + (on ? h : 0)) * a.R);
    const T* qr = reinterpret_cast<const T*>(a.qkv) + (int64_t)m * a.ldq + (int64_t)(on ? h : 0) * (a.dim + a.rd) + a.dim;
    for (int v = lane; v < a.R / 8; v += 32)
      reinterpret_cast<uint4*>(sQ + r * ld)[v] = on ? qv[v] : make_uint4(0, 0, 0, 0);
    for (int i = lane; i < Dp - a.R; i += 32) sQ[r * ld + a.R + i] = on && i < a.rd ? qr[i] : DT<T>::from_f(0.f);
  }
  __syncthreads();
  uint32_t qa[KS][4];
#pragma unroll
  for (int s = 0; s < KS; ++s)
    if (s < ks) ldsm4(qa[s], sQ + (mg * 16 + ar) * ld + k0 + s * 16 + ac);
  float o[MG][RT][4] = {};
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};     // rows warp * 2 + i of the CTA
  for (int t = 0; t < ntile; ++t) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 2) : "memory");
    __syncthreads();                              // tile t is in; everybody is done with tile t - 1
    if (t + kStages - 1 < ntile) load_tile(t + kStages - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const T* K = sK + (t % kStages) * kKT * ld;
    {
      float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
      // matrices of one x4: keys 0-7 at k and k + 8, keys 8-15 at k and k + 8
      const T* kb = K + (kh * 16 + (lane & 7) + ((lane >> 4) << 3)) * ld + k0 + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int s = 0; s < KS; ++s) {
        if (s < ks) {
          uint32_t b[4];
          ldsm4(b, kb + s * 16);
          mma16816<T>(c0, qa[s], b[0], b[1]);
          mma16816<T>(c1, qa[s], b[2], b[3]);
        }
      }
      float* s0 = sS + ((size_t)kq * kHeads + mg * 16 + g) * kLdS + kh * 16 + tq * 2;
      *reinterpret_cast<float2*>(s0) = make_float2(c0[0], c0[1]);
      *reinterpret_cast<float2*>(s0 + 8) = make_float2(c1[0], c1[1]);
      *reinterpret_cast<float2*>(s0 + 8 * kLdS) = make_float2(c0[2], c0[3]);
      *reinterpret_cast<float2*>(s0 + 8 * kLdS + 8) = make_float2(c1[2], c1[3]);
    }
    __syncthreads();
    const bool valid = lo + t * kKT + lane < hi;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = warp * 2 + i;
      const float* sr = sS + (size_t)r * kLdS + lane;
      const float sum = (sr[0] + sr[kHeads * kLdS]) + (sr[2 * kHeads * kLdS] + sr[3 * kHeads * kLdS]);
      const float s = valid ? sum * a.scale_log2 : -INFINITY;
      const float mn = fmaxf(mrow[i], warp_max(s));
      const float corr = ex2(mrow[i] - mn);       // first tile: 2^-inf = 0
      const float p = valid ? ex2(s - mn) : 0.f;
      lrow[i] = lrow[i] * corr + warp_sum(p);
      mrow[i] = mn;
      sP[r * (kKT + 8) + lane] = DT<T>::from_f(p);
      if (lane == 0) sC[r] = corr;
    }
    __syncthreads();
    uint32_t p[MG][2][4];
    float f[MG][2];
#pragma unroll
    for (int i = 0; i < MG; ++i) {
      const T* pb = sP + (i * 16 + ar) * (kKT + 8) + ac;
      ldsm4(p[i][0], pb);
      ldsm4(p[i][1], pb + 16);
      f[i][0] = sC[i * 16 + g];
      f[i][1] = sC[i * 16 + g + 8];
    }
#pragma unroll
    for (int j = 0; j < RT; ++j) {
      const int n = (warp + kWarpsHere * j) * 8;
      if (n < a.R) {
        uint32_t b[4];
        ldsm4t(b, K + lane * ld + n);
#pragma unroll
        for (int i = 0; i < MG; ++i) {
          o[i][j][0] *= f[i][0]; o[i][j][1] *= f[i][0]; o[i][j][2] *= f[i][1]; o[i][j][3] *= f[i][1];
          mma16816<T>(o[i][j], p[i][0], b[0], b[1]);
          mma16816<T>(o[i][j], p[i][1], b[2], b[3]);
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  const int64_t part0 = ((int64_t)m * a.nsplit + split) * a.H;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int h = h0 + warp * 2 + i;
    if (lane == 0 && h < a.H) {
      a.ml[(part0 + h) * 2] = mrow[i];
      a.ml[(part0 + h) * 2 + 1] = lrow[i];
    }
  }
  if (ntile == 0) return;                         // l = 0: the merge does not read this split's output
#pragma unroll
  for (int j = 0; j < RT; ++j) {
    const int n = (warp + kWarpsHere * j) * 8 + tq * 2;
    if (n < a.R) {
#pragma unroll
      for (int i = 0; i < MG; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int h = h0 + i * 16 + g + 8 * e;
          if (h < a.H)
            *reinterpret_cast<float2*>(a.o + (part0 + h) * a.R + n) = make_float2(o[i][j][2 * e], o[i][j][2 * e + 1]);
        }
    }
  }
}

template <typename T, int MG, int RT, int KS>
cudaError_t launch_mma(const LatentAttnArgs& a, bool pdl, cudaStream_t st) {
  auto kern = latent_attn_mma_kernel<T, MG, RT, KS>;
  const size_t ld = (size_t)a.ldc + 8;
  const size_t smem = sizeof(T) * (kStages * kKT * ld + MG * 16 * (kKT + 8)) +
                      sizeof(float) * (4 * MG * 16 * (kKT + 4) + MG * 16);
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  dim3 grid((a.H + MG * 16 - 1) / (MG * 16), a.nsplit, a.M);
  return launch_kernel(kern, grid, dim3(MG * 256), smem, st, pdl, a);
}

template <typename T, int MG>
cudaError_t dispatch_rt(const LatentAttnArgs& a, bool pdl, cudaStream_t st) {
  if (a.R <= 128 && a.ldc <= 320) return launch_mma<T, MG, 2 / MG, 5>(a, pdl, st);
  if (a.R <= 256 && a.ldc <= 320) return launch_mma<T, MG, 4 / MG, 5>(a, pdl, st);
  return launch_mma<T, MG, 8 / MG, 10>(a, pdl, st);
}

// ------------------------------------------------------------------------------------------------ merge + W_uv
struct UvArgs {
  const float* o;
  const float* ml;
  const void* w_uv;     // T [H * vd, R]
  void* out;            // T [M, ldo], head h at h * vd
  int64_t ldo;
  int M, H, R, vd, nsplit, rows_per_block;
  const void* gate;     // T [M, ldg], head h at h * vd, or null: outputs times sigmoid(gate)
  int64_t ldg;
};

constexpr int kUvThreads = 256;
template <typename T, int V, int MT>
__global__ void __launch_bounds__(kUvThreads) latent_uv_kernel(UvArgs a) {
  extern __shared__ __align__(16) float sh[];   // [MT][R4] merged latents, [MT][nsplit] weights
  __shared__ int s_valid[MT];
  const int R4 = (a.R + 3) / 4 * 4;
  float* so = sh;
  float* sw = sh + MT * R4;
  const int h = blockIdx.x, m0 = blockIdx.z * MT, mn = min(MT, a.M - m0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (warp < MT) {                              // a warp per token: weights of the splits (empty ones come last)
    const int m = m0 + warp;
    float* w = sw + warp * a.nsplit;
    int nv = 0;
    if (warp < mn) {
      float mx = -INFINITY, l = 0.f;
      for (int s = lane; s < a.nsplit; s += 32) {
        const float* e = a.ml + (((int64_t)m * a.nsplit + s) * a.H + h) * 2;
        if (e[1] > 0.f) { mx = fmaxf(mx, e[0]); nv = s + 1; }
      }
      mx = warp_max(mx);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) nv = max(nv, __shfl_xor_sync(0xffffffffu, nv, o));
      for (int s = lane; s < a.nsplit; s += 32) {
        const float* e = a.ml + (((int64_t)m * a.nsplit + s) * a.H + h) * 2;
        const float f = e[1] > 0.f ? exp2f(e[0] - mx) : 0.f;
        w[s] = f;
        l += f * e[1];
      }
      l = warp_sum(l);
      const float inv = l > 0.f ? 1.0f / l : 0.f;
      for (int s = lane; s < a.nsplit; s += 32) w[s] *= inv;
    }
    if (lane == 0) s_valid[warp] = nv;
  }
  __syncthreads();
#pragma unroll
  for (int mm = 0; mm < MT; ++mm) {
    const int nv = s_valid[mm];
    const float* w = sw + mm * a.nsplit;
    const float* src = a.o + ((int64_t)(m0 + mm) * a.nsplit * a.H + h) * a.R;
    const int64_t step = (int64_t)a.H * a.R;
    if (a.R % 2 == 0) {
      for (int r = threadIdx.x * 2; r < a.R; r += kUvThreads * 2) {
        float2 v = make_float2(0.f, 0.f);
        for (int s0 = 0; s0 < nv; s0 += 16) {          // sixteen partial rows in flight
          float2 x[16];
#pragma unroll
          for (int i = 0; i < 16; ++i)
            x[i] = s0 + i < nv ? *reinterpret_cast<const float2*>(src + (s0 + i) * step + r) : make_float2(0.f, 0.f);
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float f = s0 + i < nv ? w[s0 + i] : 0.f;
            v.x = fmaf(f, x[i].x, v.x);
            v.y = fmaf(f, x[i].y, v.y);
          }
        }
        so[mm * R4 + r] = v.x;
        so[mm * R4 + r + 1] = v.y;
      }
    } else {
      for (int r = threadIdx.x; r < a.R; r += kUvThreads) {
        float v = 0.f;
        for (int s = 0; s < nv; ++s) v = fmaf(w[s], src[s * step + r], v);
        so[mm * R4 + r] = v;
      }
    }
  }
  __syncthreads();
  constexpr int RW = 4;                          // value rows a warp works on at a time
  const int v0 = blockIdx.y * a.rows_per_block, v1 = min(v0 + a.rows_per_block, a.vd);
  for (int v = v0 + warp * RW; v < v1; v += kUvThreads / 32 * RW) {
    const T* w = reinterpret_cast<const T*>(a.w_uv) + ((int64_t)h * a.vd + v) * a.R;
    float acc[RW][MT] = {};
    for (int r = lane * V; r < a.R; r += 32 * V) {
      float wf[RW][V];
#pragma unroll
      for (int q = 0; q < RW; ++q) {
        const T* wq = w + (int64_t)min(q, v1 - 1 - v) * a.R + r;
        if constexpr (V > 1) {
          const uint4 raw = ldg_nc_v4(wq);
          const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
          for (int i = 0; i < V; ++i) wf[q][i] = DT<T>::to_f(e[i]);
        } else {
          wf[q][0] = DT<T>::to_f(*wq);
        }
      }
#pragma unroll
      for (int mm = 0; mm < MT; ++mm)
#pragma unroll
        for (int i = 0; i < V; ++i) {
          const float x = so[mm * R4 + r + i];
#pragma unroll
          for (int q = 0; q < RW; ++q) acc[q][mm] = fmaf(x, wf[q][i], acc[q][mm]);
        }
    }
#pragma unroll
    for (int q = 0; q < RW; ++q)
#pragma unroll
      for (int mm = 0; mm < MT; ++mm) {
        float s = warp_sum(acc[q][mm]);
        if (lane == q * MT + mm && mm < mn && v + q < v1) {
          if (a.gate != nullptr)
            s /= 1.0f + expf(-DT<T>::to_f(reinterpret_cast<const T*>(a.gate)[(int64_t)(m0 + mm) * a.ldg + (int64_t)h * a.vd + v + q]));
          reinterpret_cast<T*>(a.out)[(int64_t)(m0 + mm) * a.ldo + (int64_t)h * a.vd + v + q] = DT<T>::from_f(s);
        }
      }
  }
}

template <typename K>
cudaError_t allow_smem(K kern, size_t smem) {
  if (smem <= 40 * 1024) return cudaSuccess;      // static shared memory counts against the default limit too
  if (smem > 226 * 1024) return cudaErrorInvalidValue;
  return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

template <typename T, int V, int MT>
cudaError_t launch_prep(const PrepArgs& a, bool pdl, cudaStream_t st) {
  auto kern = latent_prep_kernel<T, V, MT>;
  const size_t smem = (size_t)MT * a.dim * sizeof(float);
  cudaError_t e = allow_smem(kern, smem);
  if (e != cudaSuccess) return e;
  const int cb = (a.R + kPrepCols - 1) / kPrepCols;
  return launch_kernel(kern, dim3(a.H * cb + (a.kv != nullptr), (a.M + MT - 1) / MT), dim3(kPrepThreads), smem, st, pdl, a);
}

template <typename T, int V, int MT>
cudaError_t launch_uv(UvArgs& a, int blocks_y, bool pdl, cudaStream_t st) {
  auto kern = latent_uv_kernel<T, V, MT>;
  const size_t smem = (size_t)MT * ((a.R + 3) / 4 * 4 + a.nsplit) * sizeof(float);
  cudaError_t e = allow_smem(kern, smem);
  if (e != cudaSuccess) return e;
  return launch_kernel(kern, dim3(a.H, blocks_y, (a.M + MT - 1) / MT), dim3(kUvThreads), smem, st, pdl, a);
}

}  // namespace

// Before the absorbed attention of M query tokens; see PrepArgs (kv null: queries only).  half: rotated pairs (2 * half <= rd).
IPEX_API int ipex_latent_prep(void* q, int64_t ldq, const void* kv, int64_t ldkv, const void* norm_w, float eps, const void* w_uk, const float* cosp,
                              const float* sinp, const int* slot, const int* pos, const int* start, void* cache,
                              int64_t slot_stride, int64_t ldc, void* qabs, int M, int H, int dim, int rd, int R,
                              int half, int dtype, int pdl, void* stream) {
  if (M < 1 || M > 65535 || H < 1 || dim < 1 || rd < 0 || R < 1 || half < 0 || 2 * half > rd || ldc < R + rd)
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    PrepArgs a = {q, kv, norm_w, w_uk, cosp, sinp, slot, pos, start, cache, qabs, nullptr, nullptr, ldq, ldkv, slot_stride, ldc,
                  0, 0, eps, M, H, dim, rd, R, half};
    cudaStream_t st = (cudaStream_t)stream;
    const bool vec = R % Vec<T>::n == 0 && (reinterpret_cast<uintptr_t>(w_uk) & 15) == 0;
    if (M == 1) return vec ? launch_prep<T, Vec<T>::n, 1>(a, pdl, st) : launch_prep<T, 1, 1>(a, pdl, st);
    return vec ? launch_prep<T, Vec<T>::n, 4>(a, pdl, st) : launch_prep<T, 1, 4>(a, pdl, st);
  });
}

// Before the prompt attention: rotates the queries in place, appends to the cache, writes contiguous latents
// c_out [M, ld_c] and rotated key parts kr_out [M, ld_kr] (kv null: the queries only).
IPEX_API int ipex_latent_prompt_prep(void* q, int64_t ldq, const void* kv, int64_t ldkv, const void* norm_w, float eps, const float* cosp,
                                     const float* sinp, const int* slot, const int* pos, const int* start, void* cache,
                                     int64_t slot_stride, int64_t ldc, void* c_out, int64_t ld_c, void* kr_out,
                                     int64_t ld_kr, int M, int H, int dim, int rd, int R, int half, int dtype, int pdl,
                                     void* stream) {
  if (M < 1 || H < 1 || dim < 1 || rd < 0 || R < 1 || half < 0 || 2 * half > rd || ldc < R + rd ||
      (kv != nullptr && (ld_c < R || ld_kr < rd)))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    PrepArgs a = {q, kv, norm_w, nullptr, cosp, sinp, slot, pos, start, cache, nullptr, c_out, kr_out, ldq, ldkv, slot_stride,
                  ldc, ld_c, ld_kr, eps, M, H, dim, rd, R, half};
    return launch_kernel(latent_prompt_prep_kernel<T>, dim3(M), dim3(256), 0, (cudaStream_t)stream, pdl != 0, a);
  });
}

// Cache row stride (elements) the attention kernels want for R + rd values.
IPEX_API int ipex_latent_row(int R, int rd, int dtype) {
  const int a = dtype == DT_F32 ? 4 : 64;
  return (R + rd + a - 1) / a * a;
}

// Whether the tensor-core kernel takes the sizes (the generic one takes all).
IPEX_API int ipex_latent_attn_fast(int R, int rd, int dtype) {
  return dtype != DT_F32 && R % 8 == 0 && R <= 512 && R + rd <= 640;
}

// Partial attention of M query tokens over the cache rows in [max(start, pos - window + 1), pos] (window 0: all),
// split in nsplit parts: o [M, nsplit, H, R] and ml [M, nsplit, H, 2] in fp32.  force_generic: 1 takes the generic
// kernel.
IPEX_API int ipex_latent_attn(const void* qabs, const void* qkv, int64_t ldq, const void* cache, int64_t slot_stride,
                              int64_t ldc, const int* slot, const int* pos, const int* start, float* o, float* ml, int M,
                              int H, int dim, int rd, int R, int window, int nsplit, float scale, int force_generic,
                              int dtype, int pdl, void* stream) {
  if (M < 1 || M > 65535 || H < 1 || R < 1 || rd < 0 || nsplit < 1 || nsplit > 65535 || window < 0 || ldc < R + rd)
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    LatentAttnArgs a = {qabs, qkv, cache, slot, pos, start, o, ml, ldq, slot_stride, ldc, scale * 1.4426950408889634f,
                        M, H, dim, rd, R, window, nsplit};
    cudaStream_t st = (cudaStream_t)stream;
    if constexpr (sizeof(T) == 2) {
      if (!force_generic && ipex_latent_attn_fast(R, rd, dtype) && ldc == ipex_latent_row(R, rd, dtype) &&
          slot_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(cache) & 15) == 0)
        return H <= 16 ? dispatch_rt<T, 1>(a, pdl != 0, st) : dispatch_rt<T, 2>(a, pdl != 0, st);
    }
    const size_t smem = ((size_t)R + rd + (size_t)kGenWarps * R) * sizeof(float);
    cudaError_t e = allow_smem(latent_attn_generic_kernel<T>, smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(latent_attn_generic_kernel<T>, dim3(H, nsplit, M), dim3(kGenWarps * 32), smem, st, pdl != 0, a);
  });
}

// out[m, h * vd + v] = W_uv[h * vd + v] . (merged latent output of head h), times sigmoid(gate [M, ldg]) unless gate is null
IPEX_API int ipex_latent_uv(const float* o, const float* ml, const void* w_uv, const void* gate, int64_t ldg, void* out,
                            int64_t ldo, int M, int H,
                            int R, int vd, int nsplit, int dtype, int pdl, void* stream) {
  if (M < 1 || H < 1 || R < 1 || vd < 1 || nsplit < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int mt = M == 1 ? 1 : 4;
    if ((M + mt - 1) / mt > 65535) return cudaErrorInvalidValue;
    // enough blocks for the machine, at least four rows per warp each
    const int have = H * ((M + mt - 1) / mt);
    int by = (296 + have - 1) / have;
    const int most = (vd + 31) / 32;
    by = by < 1 ? 1 : (by > most ? most : by);
    UvArgs a = {o, ml, w_uv, out, ldo, M, H, R, vd, nsplit, (vd + by - 1) / by, gate, ldg};
    cudaStream_t st = (cudaStream_t)stream;
    const bool vec = R % Vec<T>::n == 0 && (reinterpret_cast<uintptr_t>(w_uv) & 15) == 0;
    if (mt == 1) return vec ? launch_uv<T, Vec<T>::n, 1>(a, by, pdl, st) : launch_uv<T, 1, 1>(a, by, pdl, st);
    return vec ? launch_uv<T, Vec<T>::n, 4>(a, by, pdl, st) : launch_uv<T, 1, 4>(a, by, pdl, st);
  });
}
