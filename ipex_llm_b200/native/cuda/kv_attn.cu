// Attention over cached keys and values of different sizes, sm_100a: everything earlier, a sliding window - alone or beside
// pooled blocks of what has left it - or the query's own chunk of positions, with an optional sink (a score of 0 or one
// learned number per head), mixed values, rotated and (unit- or weighted-) normed queries and keys, and gated outputs.
//
//   qk_prepare  norm and rotation of the query and key heads of many tokens in place (prompts, portions)
//   kv_append   keys and values of the new tokens into the cache, the values mixed with those of an earlier layer;
//               for prompts also the transposed values that the tcgen05 prompt attention reads
//   kv_pool     means of the keys and values of the blocks of tokens that a portion completes, into the cache's rows of
//               blocks and, for prompts, where the prompt attention reads them
//   kv_attn     attention of query tokens against what their slots hold: decoding (which prepares and appends its own
//               row on the way), portions of prompts, and whole prompts of sizes or formats the tensor-core kernel does not take
//
// kv_attn: a cluster of up to eight CTAs shares the visible keys of one query token for up to RT query heads of one key
// head.  A CTA walks its keys in tiles: eight lanes share a key for the scores (every lane has four keys in flight), the
// tile's weights meet in shared memory, then threads own value columns and take turns over the keys.  The parts of a
// cluster are merged through distributed shared memory, where the sink joins the denominator; nothing but the output is
// written, so the step needs no scratch and no second launch.
#include <cooperative_groups.h>

#include "common/utils.cuh"

namespace {

namespace cg = cooperative_groups;

constexpr int kThreads = 256;
constexpr int kTile = 128;            // keys per tile

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

// 16 bytes (VN elements) or a single element
template <typename T, bool VEC> struct Pack {
  static constexpr int n = VEC ? 16 / (int)sizeof(T) : 1;
};

template <typename T, bool VEC>
__device__ __forceinline__ void load_pack(const T* p, float (&f)[Pack<T, VEC>::n]) {
  if constexpr (!VEC) {
    f[0] = DT<T>::to_f(*p);
  } else {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
    for (int i = 0; i < Pack<T, VEC>::n; ++i) f[i] = DT<T>::to_f(e[i]);
  }
}

__device__ __forceinline__ float mixed(float v, float first, float lambda) { return (1.0f - lambda) * v + lambda * first; }

// ---------------------------------------------------------------------------------------------- rotation and unit norm
struct Prepare {
  const float* cosp;    // [positions, half], row = position in the sequence
  const float* sinp;
  int half;             // pairs (i, i + half) of a head turn
  int unit;             // divide by the root mean square
  float eps;
  const float* wq;      // [dim] weight of the queries' norm, or null
  const float* wk;      // ... and of the keys'
  int q_heads;          // heads of x that are queries (qk_prepare)
};

// One vector by one warp; load(i) / store(i, value) for its elements.  The norm comes before the rotation, which does not
// change it; every lane finishes its own pairs.  w: weight of the norm, or null.
template <typename L, typename S>
__device__ __forceinline__ void prepare_vector(const Prepare& p, int dim, int rel, float scale, int lane, const float* w,
                                               L&& load, S&& store) {
  float f = scale;
  if (p.unit) {
    float ss = 0.f;
    for (int i = lane; i < dim; i += 32) {
      const float x = load(i);
      ss = fmaf(x, x, ss);
    }
    f = scale / sqrtf(warp_sum(ss) / (float)dim + p.eps);
  }
  const float* cp = p.cosp + (int64_t)rel * p.half;
  const float* sp = p.sinp + (int64_t)rel * p.half;
  auto at = [&](int i) { return w != nullptr ? load(i) * w[i] : load(i); };
  for (int i = lane; i < p.half; i += 32) {
    const float u = at(i), v = at(i + p.half), c = cp[i], s = sp[i];
    store(i, (u * c - v * s) * f);
    store(i + p.half, (v * c + u * s) * f);
  }
  for (int i = 2 * p.half + lane; i < dim; i += 32) store(i, at(i) * f);
}

// A warp per (token, head) of x: rows of `ld`, heads behind one another.
template <typename T>
__global__ void __launch_bounds__(kThreads) qk_prepare_kernel(T* __restrict__ x, int64_t ld, const int* __restrict__ slot,
                                                              const int* __restrict__ pos, const int* __restrict__ start,
                                                              Prepare p, int64_t rows, int heads, int dim) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t r = (int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int t = (int)(r / heads), h = (int)(r % heads);
  T* v = x + (int64_t)t * ld + (int64_t)h * dim;
  prepare_vector(p, dim, pos[t] - start[slot[t]], 1.0f, threadIdx.x & 31, h < p.q_heads ? p.wq : p.wk,
                 [&](int i) { return DT<T>::to_f(v[i]); },
                 [&](int i, float y) { v[i] = DT<T>::from_f(y); });
}

// The same 16 bytes at a time: LG lanes hold a head, a pack each (dim <= LG packs), partners meet in shuffles; a group works
// on kHeads heads at once, whose loads are all in flight together.
template <typename T, int LG>
__global__ void __launch_bounds__(kThreads) qk_prepare_vec_kernel(T* __restrict__ x, int64_t ld, const int* __restrict__ slot,
                                                                  const int* __restrict__ pos, const int* __restrict__ start,
                                                                  Prepare p, uint32_t rows, uint32_t heads, int dim) {
  constexpr int N = Pack<T, true>::n, kHeads = 4;
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t r0 = (blockIdx.x * (kThreads / LG) + threadIdx.x / LG) * kHeads;
  const int lane = threadIdx.x % LG, hp = p.half / N;
  const bool mine = lane * N < dim, first = lane < hp, turns = lane < 2 * hp;
  T* v[kHeads];
  const float* wt[kHeads];
  float a[kHeads][N];
  int64_t at[kHeads];
#pragma unroll
  for (int u = 0; u < kHeads; ++u) {
    const uint32_t r = r0 + u, t = r < rows ? r / heads : 0, h = r < rows ? r - t * heads : 0;
    v[u] = x + (int64_t)t * ld + (int64_t)h * dim + lane * N;
    wt[u] = h < (uint32_t)p.q_heads ? p.wq : p.wk;
    at[u] = (int64_t)(pos[t] - start[slot[t]]) * p.half + (first ? lane : lane - hp) * N;
#pragma unroll
    for (int j = 0; j < N; ++j) a[u][j] = 0.f;
    if (r < rows && mine) load_pack<T, true>(v[u], a[u]);
  }
#pragma unroll
  for (int u = 0; u < kHeads; ++u) {
    float f = 1.f;
    if (p.unit) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < N; ++j) ss = fmaf(a[u][j], a[u][j], ss);
#pragma unroll
      for (int o = LG / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      f = 1.0f / sqrtf(ss / (float)dim + p.eps);
    }
    if (wt[u] != nullptr && mine) {
#pragma unroll
      for (int j = 0; j < N; ++j) a[u][j] *= wt[u][lane * N + j];
    }
    float b[N];
    const int partner = !turns ? lane : first ? lane + hp : lane - hp;
#pragma unroll
    for (int j = 0; j < N; ++j) b[j] = __shfl_sync(0xffffffffu, a[u][j], partner, LG);
    if (r0 + u < rows && mine) {
      if (turns) {
        const float sign = first ? -1.f : 1.f;
#pragma unroll
        for (int j = 0; j < N; j += 4) {
          const float4 c = *reinterpret_cast<const float4*>(p.cosp + at[u] + j);
          const float4 s = *reinterpret_cast<const float4*>(p.sinp + at[u] + j);
          const float cs[4] = {c.x, c.y, c.z, c.w}, sn[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) a[u][j + e] = a[u][j + e] * cs[e] + sign * b[j + e] * sn[e];
        }
      }
      __align__(16) T o[N];
#pragma unroll
      for (int j = 0; j < N; ++j) o[j] = DT<T>::from_f(a[u][j] * f);
      *reinterpret_cast<uint4*>(v[u]) = *reinterpret_cast<const uint4*>(o);
    }
  }
}

template <typename T, int LG>
cudaError_t launch_prepare(void* x, int64_t ld, const int* slot, const int* pos, const int* start, const Prepare& p,
                           int64_t rows, int heads, int dim, bool pdl, cudaStream_t st) {
  const int64_t per = (int64_t)kThreads / LG * 4;
  return launch_kernel(qk_prepare_vec_kernel<T, LG>, dim3((unsigned)((rows + per - 1) / per)), dim3(kThreads), 0, st, pdl,
                       (T*)x, ld, slot, pos, start, p, (uint32_t)rows, (uint32_t)heads, dim);
}

// ---------------------------------------------------------------------------------------------- append
struct AppendArgs {
  const void* k;        // T [tokens, ld] at head * dim
  const void* v;        // T [tokens, ld] at head * vdim
  const void* vfirst;   // T [tokens, ld_vf] or null
  void* kc;             // cache rows: slot * k_slot + head * k_head + position * dim
  void* vc;
  void* vt;             // T [heads * vdim, ld_vt] or null
  const int* slot;
  const int* pos;
  int64_t ld, ld_vf, k_slot, k_head, v_slot, v_head, ld_vt;
  float lambda;
  int tokens, dim, vdim;
};

// CTA = 64 tokens of one head.
template <typename T>
__global__ void __launch_bounds__(kThreads) kv_append_kernel(AppendArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  T* sv = reinterpret_cast<T*>(smem);              // [64][vdim + pad] when vt is wanted
  const int t0 = blockIdx.x * 64, g = blockIdx.y, nt = min(64, a.tokens - t0);
  const int ldsv = (a.vdim + 1) | 1;               // odd: columns fall into different banks
  pdl_launch_dependents();
  pdl_wait();
  const T* k = reinterpret_cast<const T*>(a.k);
  const T* v = reinterpret_cast<const T*>(a.v);
  const T* vf = reinterpret_cast<const T*>(a.vfirst);
  T* kc = reinterpret_cast<T*>(a.kc);
  T* vc = reinterpret_cast<T*>(a.vc);
  constexpr int VN = 16 / (int)sizeof(T);
  const bool kvec = a.dim % VN == 0 && a.ld % VN == 0 && (((uintptr_t)k | (uintptr_t)kc) & 15) == 0;
  if (kvec) {
    const int nv = a.dim / VN;
    for (int i = threadIdx.x; i < nt * nv; i += kThreads) {
      const int t = i / nv, c = i % nv;
      const uint4 x = *reinterpret_cast<const uint4*>(k + (int64_t)(t0 + t) * a.ld + (int64_t)g * a.dim + c * VN);
      T* row = kc + (int64_t)a.slot[t0 + t] * a.k_slot + (int64_t)g * a.k_head + (int64_t)a.pos[t0 + t] * a.dim;
      *reinterpret_cast<uint4*>(row + c * VN) = x;
    }
  } else {
    for (int i = threadIdx.x; i < nt * a.dim; i += kThreads) {
      const int t = i / a.dim, c = i % a.dim;
      kc[(int64_t)a.slot[t0 + t] * a.k_slot + (int64_t)g * a.k_head + (int64_t)a.pos[t0 + t] * a.dim + c] =
          k[(int64_t)(t0 + t) * a.ld + (int64_t)g * a.dim + c];
    }
  }
  const bool vvec = a.vdim % VN == 0 && a.ld % VN == 0 && (((uintptr_t)v | (uintptr_t)vc) & 15) == 0 &&
                    (vf == nullptr || (a.ld_vf % VN == 0 && ((uintptr_t)vf & 15) == 0));
  auto values = [&](auto tag) {
    constexpr bool VEC = decltype(tag)::value;
    constexpr int N = Pack<T, VEC>::n;
    const int nv = a.vdim / N;
    for (int i = threadIdx.x; i < nt * nv; i += kThreads) {
      const int t = i / nv, c = (i % nv) * N;
      float x[N];
      load_pack<T, VEC>(v + (int64_t)(t0 + t) * a.ld + (int64_t)g * a.vdim + c, x);
      if (vf != nullptr) {
        float y[N];
        load_pack<T, VEC>(vf + (int64_t)(t0 + t) * a.ld_vf + (int64_t)g * a.vdim + c, y);
#pragma unroll
        for (int j = 0; j < N; ++j) x[j] = mixed(x[j], y[j], a.lambda);
      }
      __align__(16) T o[N];
#pragma unroll
      for (int j = 0; j < N; ++j) o[j] = DT<T>::from_f(x[j]);
      T* row = vc + (int64_t)a.slot[t0 + t] * a.v_slot + (int64_t)g * a.v_head + (int64_t)a.pos[t0 + t] * a.vdim + c;
      if constexpr (VEC) *reinterpret_cast<uint4*>(row) = *reinterpret_cast<const uint4*>(o);
      else row[0] = o[0];
      if (a.vt != nullptr) {
#pragma unroll
        for (int j = 0; j < N; ++j) sv[t * ldsv + c + j] = o[j];
      }
    }
  };
  if (vvec) values(std::true_type{});
  else values(std::false_type{});
  if (a.vt == nullptr) return;
  __syncthreads();
  // ld_vt is a multiple of VN, so whole vectors of tokens always fit; tokens past the end are zero
  T* vt = reinterpret_cast<T*>(a.vt);
  constexpr int TV = 64 / VN;
  for (int i = threadIdx.x; i < a.vdim * TV; i += kThreads) {
    const int c = i / TV, t = (i % TV) * VN;
    if (t >= nt) continue;
    __align__(16) T o[VN];
#pragma unroll
    for (int j = 0; j < VN; ++j) o[j] = t + j < nt ? sv[(t + j) * ldsv + c] : DT<T>::from_f(0.f);
    *reinterpret_cast<uint4*>(vt + (int64_t)(g * a.vdim + c) * a.ld_vt + t0 + t) = *reinterpret_cast<const uint4*>(o);
  }
}

// ---------------------------------------------------------------------------------------------- pooled blocks
struct PoolArgs {
  const void* kc;       // cache rows: slot * k_slot + head * k_head + position * dim
  const void* vc;
  void* pk;             // rows of blocks: slot * pk_slot + head * pk_head + block * dim
  void* pv;
  void* kp;             // prompts: T [rows, ld_kp], head h at h * dim, rows from pool_row[portion] on; or null
  void* vt;             // ... and T [heads * vdim, ld_vt]
  const int* slot;      // [tokens]
  const int* pos;       // [tokens]
  const int* start;     // [slots]
  const int* seq_row;   // [portions]
  const int* seq_len;   // [portions]
  const int* pool_row;  // [portions], or null
  int64_t k_slot, k_head, v_slot, v_head, pk_slot, pk_head, pv_slot, pv_head, ld_kp, ld_vt;
  int pool, dim, vdim;
};

// Mean of a block's rows, in order; what the attention of a decoded token computes for the block it completes.
template <typename T>
__device__ __forceinline__ T block_mean(const T* rows, int dim, int pool) {
  float s = 0.f;
#pragma unroll 4
  for (int j = 0; j < pool; ++j) s += DT<T>::to_f(rows[(int64_t)j * dim]);
  return DT<T>::from_f(s / (float)pool);
}

// A warp per (block, head, portion).
template <typename T>
__global__ void __launch_bounds__(kThreads) kv_pool_kernel(PoolArgs a) {
  const int seq = blockIdx.z, g = blockIdx.y, lane = threadIdx.x & 31;
  const int row0 = a.seq_row[seq], len = a.seq_len[seq], slot = a.slot[row0], start = a.start[slot];
  const int p0 = a.pos[row0] - start, b = p0 / a.pool + blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  if ((int64_t)(b + 1) * a.pool > p0 + len) return;
  const int64_t first = start + (int64_t)b * a.pool;
  const T* k = reinterpret_cast<const T*>(a.kc) + slot * a.k_slot + g * a.k_head + first * a.dim;
  const T* v = reinterpret_cast<const T*>(a.vc) + slot * a.v_slot + g * a.v_head + first * a.vdim;
  T* pk = reinterpret_cast<T*>(a.pk) + slot * a.pk_slot + g * a.pk_head + (int64_t)b * a.dim;
  T* pv = reinterpret_cast<T*>(a.pv) + slot * a.pv_slot + g * a.pv_head + (int64_t)b * a.vdim;
  const int64_t row = a.pool_row != nullptr ? a.pool_row[seq] + b : 0;
  for (int i = lane; i < a.dim; i += 32) {
    const T m = block_mean(k + i, a.dim, a.pool);
    pk[i] = m;
    if (a.kp != nullptr) reinterpret_cast<T*>(a.kp)[row * a.ld_kp + (int64_t)g * a.dim + i] = m;
  }
  for (int i = lane; i < a.vdim; i += 32) {
    const T m = block_mean(v + i, a.vdim, a.pool);
    pv[i] = m;
    if (a.vt != nullptr) reinterpret_cast<T*>(a.vt)[((int64_t)g * a.vdim + i) * a.ld_vt + row] = m;
  }
}

// ---------------------------------------------------------------------------------------------- attention
struct AttnArgs {
  const void* q;        // T [tokens, ldq], head h at h * dim
  const void* k;        // append: this launch's own keys and values, T [tokens, ldq] at kv head * dim / vdim
  const void* v;
  const void* vfirst;   // T [tokens, ld_vf] or null
  void* kc;
  void* vc;
  void* out;            // T [tokens, ldo], head h at h * vdim
  const int* slot;
  const int* pos;
  const int* start;     // [slots] position of the sequence's first token
  int64_t ldq, ld_vf, ldo, k_slot, k_head, v_slot, v_head;
  float lambda, scale;
  int heads, kv_heads, dim, vdim, window, sink, append;
  int chunk;            // keys of the query's own chunk of this many positions only; 0: all
  const float* sinks;   // [heads] scores of the sink; null: 0
  const void* gate;     // T [tokens, ldg], head h at h * vdim, or null: outputs times gate_scale * sigmoid(gate)
  int64_t ldg;
  float gate_scale;
  Prepare prep;
  int prepare;          // with append: queries and the new key are rotated / normed here
  int pool;             // > 0: beside the window, the blocks of this many tokens that lie wholly before it
  void* pk;             // rows of blocks: slot * pk_slot + head * pk_head + block * dim
  void* pv;
  int64_t pk_slot, pk_head, pv_slot, pv_head;
};

template <typename T, int RT, bool VEC>
__global__ void __launch_bounds__(kThreads) kv_attn_kernel(AttnArgs a, int nrb) {
  constexpr int VN = Pack<T, VEC>::n;
  extern __shared__ __align__(16) float sm[];
  cg::cluster_group cluster = cg::this_cluster();
  const int nsplit = gridDim.x, split = blockIdx.x;
  const int g = blockIdx.y / nrb, rb = blockIdx.y % nrb, tok = blockIdx.z;
  const int R = a.heads / a.kv_heads, r0 = rb * RT, rows = min(RT, R - r0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dimp = (a.dim + 3) & ~3;
  float* sq = sm;                                // [RT + 1][dimp] scaled queries, the new key
  float* ss = sq + (RT + 1) * dimp;              // [RT][kTile] scores, then weights
  float* sc = ss + RT * kTile;                   // [RT] factor of what was gathered before this tile
  float* sml = sc + RT;                          // [RT][2] maximum and sum
  float* so = sml + 2 * RT;                      // [RT][vdim] this CTA's part of the output
  float* sred = so + RT * ((a.vdim + 3) & ~3);   // [subsets][RT][vdim]
  pdl_launch_dependents();
  pdl_wait();
  const int slot = a.slot[tok], pos = a.pos[tok], start = a.start[slot];
  int lo = max(start, a.window > 0 ? pos - a.window + 1 : 0);
  if (a.chunk > 0) lo = max(lo, pos - (pos - start) % a.chunk);
  // keys 0 .. nb are blocks, the others tokens from position lo on
  const int nb = a.pool > 0 ? max(0, pos - start - a.window + 1) / a.pool : 0;
  const int n = nb + pos + 1 - lo;
  const int chunk = (n + nsplit - 1) / nsplit;
  const int j0 = min(n, split * chunk), j1 = min(n, (split + 1) * chunk);
  T* kc = reinterpret_cast<T*>(a.kc) + (int64_t)slot * a.k_slot + (int64_t)g * a.k_head;
  T* vc = reinterpret_cast<T*>(a.vc) + (int64_t)slot * a.v_slot + (int64_t)g * a.v_head;
  T* pk = reinterpret_cast<T*>(a.pk) + (int64_t)slot * a.pk_slot + (int64_t)g * a.pk_head;
  T* pv = reinterpret_cast<T*>(a.pv) + (int64_t)slot * a.pv_slot + (int64_t)g * a.pv_head;
  const bool newest = a.append && j1 == n && j0 < j1;
  if (newest) {
    // this CTA owns the newest key: it files the row and reads it back like the others (every row block of the head
    // does, with the same values)
    const T* k = reinterpret_cast<const T*>(a.k) + (int64_t)tok * a.ldq + (int64_t)g * a.dim;
    const T* v = reinterpret_cast<const T*>(a.v) + (int64_t)tok * a.ldq + (int64_t)g * a.vdim;
    const T* vf = reinterpret_cast<const T*>(a.vfirst) + (int64_t)tok * a.ld_vf + (int64_t)g * a.vdim;
    if (a.prepare) {
      if (warp == RT % (kThreads / 32)) {
        float* sk = sq + RT * dimp;
        for (int i = lane; i < a.dim; i += 32) sk[i] = DT<T>::to_f(k[i]);
        __syncwarp();
        T* dst = kc + (int64_t)pos * a.dim;
        prepare_vector(a.prep, a.dim, pos - start, 1.0f, lane, a.prep.wk, [&](int i) { return sk[i]; },
                       [&](int i, float y) { dst[i] = DT<T>::from_f(y); });
      }
    } else {
      for (int i = tid; i < a.dim; i += kThreads) kc[(int64_t)pos * a.dim + i] = k[i];
    }
    for (int i = tid; i < a.vdim; i += kThreads) {
      const float own = DT<T>::to_f(v[i]);
      vc[(int64_t)pos * a.vdim + i] =
          a.vfirst != nullptr ? DT<T>::from_f(mixed(own, DT<T>::to_f(vf[i]), a.lambda)) : v[i];
    }
  }
  {
    const T* q = reinterpret_cast<const T*>(a.q) + (int64_t)tok * a.ldq + (int64_t)(g * R + r0) * a.dim;
    if (a.prepare) {
      if (warp < RT) {
        float* dst = sq + warp * dimp;
        for (int i = lane; i < a.dim; i += 32) dst[i] = warp < rows ? DT<T>::to_f(q[(int64_t)warp * a.dim + i]) : 0.f;
        __syncwarp();
        if (warp < rows)
          prepare_vector(a.prep, a.dim, pos - start, a.scale, lane, a.prep.wq, [&](int i) { return dst[i]; },
                         [&](int i, float y) { dst[i] = y; });
      }
    } else {
      for (int i = tid; i < RT * a.dim; i += kThreads) {
        const int r = i / a.dim, c = i % a.dim;
        sq[r * dimp + c] = r < rows ? DT<T>::to_f(q[(int64_t)r * a.dim + c]) * a.scale : 0.f;
      }
    }
  }
  __syncthreads();
  if (newest && a.pool > 0 && (pos - start + 1) % a.pool == 0) {
    // the new token completes a block, which nobody sees yet
    const int b = (pos - start) / a.pool, first = start + b * a.pool;
    for (int i = tid; i < a.dim; i += kThreads)
      pk[(int64_t)b * a.dim + i] = block_mean(kc + (int64_t)first * a.dim + i, a.dim, a.pool);
    for (int i = tid; i < a.vdim; i += kThreads)
      pv[(int64_t)b * a.vdim + i] = block_mean(vc + (int64_t)first * a.vdim + i, a.vdim, a.pool);
  }

  const int nvk = a.dim / VN, nvv = a.vdim / VN;
  const int subsets = kThreads / nvv, vv = tid % nvv, sub = tid / nvv;
  const bool von = sub < subsets;
  float acc[RT][VN];
#pragma unroll
  for (int r = 0; r < RT; ++r)
#pragma unroll
    for (int i = 0; i < VN; ++i) acc[r][i] = 0.f;
  float m_row = -INFINITY, l_row = 0.f;          // of row `warp` (rows <= 8 warps)

  const int kg = lane >> 3, ks = lane & 7;       // a warp: four keys at a time, eight lanes each
  for (int t0 = j0; t0 < j1; t0 += kTile) {
    const int tn = min(kTile, j1 - t0);
    // ---- scores: warp w takes keys w * 16 .. + 15 of the tile
    if (warp * 16 < tn) {
      float s[4 * RT];
#pragma unroll
      for (int i = 0; i < 4 * RT; ++i) s[i] = 0.f;
      const T* kp[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int j = t0 + min(tn - 1, warp * 16 + u * 4 + kg);
        kp[u] = j < nb ? pk + (int64_t)j * a.dim : kc + (int64_t)(lo + j - nb) * a.dim;
      }
      for (int c = ks; c < nvk; c += 8) {
        float kf[4][VN];
#pragma unroll
        for (int u = 0; u < 4; ++u) load_pack<T, VEC>(kp[u] + c * VN, kf[u]);
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          float qf[VN];
          if constexpr (VN == 1) {
            qf[0] = sq[r * dimp + c];
          } else {
#pragma unroll
            for (int i = 0; i < VN / 4; ++i) {
              const float4 x = *reinterpret_cast<const float4*>(sq + r * dimp + c * VN + 4 * i);
              qf[4 * i] = x.x; qf[4 * i + 1] = x.y; qf[4 * i + 2] = x.z; qf[4 * i + 3] = x.w;
            }
          }
#pragma unroll
          for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int i = 0; i < VN; ++i) s[u * RT + r] = fmaf(kf[u][i], qf[i], s[u * RT + r]);
        }
      }
      // value index u * RT + r; after the folds a lane holds the block of indices its bits select
      fold<4 * RT, 4>(s, lane);
      constexpr int kKeep = 4 * RT >= 8 ? 4 * RT / 8 : 1;
      int first = 0, width = 4 * RT;
#pragma unroll
      for (int off = 4; off > 0; off >>= 1)
        if (width > 1) {
          width >>= 1;
          if (lane & off) first += width;
        }
      const bool writer = 4 * RT >= 8 || (lane & 1) == 0;        // four values on eight lanes: two lanes hold each
      if (writer) {
#pragma unroll
        for (int i = 0; i < kKeep; ++i) {
          const int idx = first + i, key = warp * 16 + idx / RT * 4 + kg;
          ss[(idx % RT) * kTile + key] = key < tn ? s[i] : -INFINITY;
        }
      }
    }
    __syncthreads();
    // ---- weights: a warp per row
    if (warp < RT) {
      float* row = ss + warp * kTile;
      float x[kTile / 32], mx = m_row;
#pragma unroll
      for (int i = 0; i < kTile / 32; ++i) {
        const int j = lane + 32 * i;
        x[i] = j < tn ? row[j] : -INFINITY;
        mx = fmaxf(mx, x[i]);
      }
      mx = warp_max(mx);
      const float ref = mx == -INFINITY ? 0.f : mx;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kTile / 32; ++i) {
        const int j = lane + 32 * i;
        const float p = x[i] == -INFINITY ? 0.f : expf(x[i] - ref);
        sum += p;
        if (j < tn) row[j] = p;
      }
      const float corr = m_row == -INFINITY ? 0.f : expf(m_row - ref);
      l_row = l_row * corr + warp_sum(sum);
      m_row = mx;
      if (lane == 0) sc[warp] = corr;
    }
    __syncthreads();
    // ---- values
    if (von) {
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        const float c = sc[r];
#pragma unroll
        for (int i = 0; i < VN; ++i) acc[r][i] *= c;
      }
      const T* vp = vc + ((int64_t)lo + t0 - nb) * a.vdim + vv * VN;
      const T* vb = pv + (int64_t)t0 * a.vdim + vv * VN;
      const int blocks = nb - t0;                // of this tile's keys
#pragma unroll 4
      for (int j = sub; j < tn; j += subsets) {
        float vf[VN];
        load_pack<T, VEC>((j < blocks ? vb : vp) + (int64_t)j * a.vdim, vf);
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          const float p = ss[r * kTile + j];
#pragma unroll
          for (int i = 0; i < VN; ++i) acc[r][i] = fmaf(p, vf[i], acc[r][i]);
        }
      }
    }
    __syncthreads();
  }
  // ---- this CTA's part
  if (von) {
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
      for (int i = 0; i < VN; ++i) sred[((size_t)sub * RT + r) * a.vdim + vv * VN + i] = acc[r][i];
  }
  if (warp < RT && lane == 0) {
    sml[2 * warp] = m_row;
    sml[2 * warp + 1] = l_row;
  }
  __syncthreads();
  for (int i = tid; i < rows * a.vdim; i += kThreads) {
    float s = 0.f;
    for (int u = 0; u < subsets; ++u) s += sred[(size_t)u * RT * a.vdim + i];
    so[i] = s;
  }
  if (nsplit > 1) cluster.sync();
  else __syncthreads();
  // ---- merge: every CTA of the cluster finishes its share of the outputs
  T* out = reinterpret_cast<T*>(a.out) + (int64_t)tok * a.ldo + (int64_t)(g * R + r0) * a.vdim;
  for (int i = split * kThreads + tid; i < rows * a.vdim; i += nsplit * kThreads) {
    const int r = i / a.vdim;
    const float zs = a.sinks != nullptr ? a.sinks[g * R + r0 + r] : 0.f;
    float m = a.sink ? zs : -INFINITY;
    for (int s = 0; s < nsplit; ++s) {
      const float* p = nsplit > 1 ? cluster.map_shared_rank(sml, s) : sml;
      m = fmaxf(m, p[2 * r]);
    }
    float l = a.sink ? expf(zs - m) : 0.f, o = 0.f;
    for (int s = 0; s < nsplit; ++s) {
      const float* p = nsplit > 1 ? cluster.map_shared_rank(sml, s) : sml;
      const float* po = nsplit > 1 ? cluster.map_shared_rank(so, s) : so;
      const float c = p[2 * r] == -INFINITY ? 0.f : expf(p[2 * r] - m);
      l = fmaf(p[2 * r + 1], c, l);
      o = fmaf(po[i], c, o);
    }
    o = l > 0.f ? o / l : 0.f;
    if (a.gate != nullptr) {
      const float z = DT<T>::to_f(reinterpret_cast<const T*>(a.gate)[(int64_t)tok * a.ldg + (int64_t)(g * R + r0) * a.vdim + i]);
      o *= a.gate_scale / (1.0f + expf(-z));
    }
    out[i] = DT<T>::from_f(o);
  }
  if (nsplit > 1) cluster.sync();      // the others may still read this CTA's part
}

template <typename T, int RT, bool VEC>
cudaError_t launch_attn(const AttnArgs& a, int tokens, int nsplit, bool pdl, cudaStream_t st) {
  constexpr int VN = Pack<T, VEC>::n;
  const int dimp = (a.dim + 3) & ~3, vp = (a.vdim + 3) & ~3, R = a.heads / a.kv_heads;
  const int nrb = (R + RT - 1) / RT, subsets = kThreads / (a.vdim / VN);
  const size_t smem = ((size_t)RT * (dimp + kTile + 3 + vp) + dimp + (size_t)subsets * RT * a.vdim + 4) * sizeof(float);
  if (smem > 220 * 1024 || (int64_t)a.kv_heads * nrb > 65535) return cudaErrorInvalidValue;
  auto kern = kv_attn_kernel<T, RT, VEC>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(nsplit, a.kv_heads * nrb, tokens);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (nsplit > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = nsplit;
    attr[na].val.clusterDim.y = 1;
    attr[na].val.clusterDim.z = 1;
    ++na;
  }
  if (pdl) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = attr;
  cfg.numAttrs = na;
  return cudaLaunchKernelEx(&cfg, kern, a, nrb);
}

template <typename T, bool VEC>
cudaError_t pick_rows(const AttnArgs& a, int tokens, int nsplit, bool pdl, cudaStream_t st) {
  const int R = a.heads / a.kv_heads;
  if (R <= 1) return launch_attn<T, 1, VEC>(a, tokens, nsplit, pdl, st);
  if (R <= 2) return launch_attn<T, 2, VEC>(a, tokens, nsplit, pdl, st);
  if (R <= 4) return launch_attn<T, 4, VEC>(a, tokens, nsplit, pdl, st);
  return launch_attn<T, 8, VEC>(a, tokens, nsplit, pdl, st);
}

}  // namespace

// Keys and values of `tokens` new tokens (k / v: rows of `ld` elements, heads behind one another) into the cache rows
// of their slots and positions; v is mixed with vfirst (may be null) by lambda.  vt (may be null): the mixed values
// transposed, [heads * vdim, ld_vt], ld_vt a multiple of 16 bytes and at least `tokens`.
IPEX_API int ipex_kv_append(const void* k, const void* v, int64_t ld, const void* vfirst, int64_t ld_vf, float lambda,
                            void* kc, int64_t k_slot, int64_t k_head, void* vc, int64_t v_slot, int64_t v_head, void* vt,
                            int64_t ld_vt, const int* slot, const int* pos, int tokens, int kv_heads, int dim, int vdim,
                            int dtype, int pdl, void* stream) {
  if (tokens < 1 || kv_heads < 1 || kv_heads > 65535 || dim < 1 || vdim < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    constexpr int VN = 16 / (int)sizeof(T);
    if (vt != nullptr && (ld_vt % VN || ld_vt < tokens || ((uintptr_t)vt & 15))) return cudaErrorInvalidValue;
    AppendArgs a = {k, v, vfirst, kc, vc, vt, slot, pos, ld, ld_vf, k_slot, k_head, v_slot, v_head, ld_vt, lambda,
                    tokens, dim, vdim};
    const size_t smem = vt != nullptr ? (size_t)64 * (vdim + 2) * sizeof(T) : 0;
    if (smem > 220 * 1024) return cudaErrorInvalidValue;
    auto kern = kv_append_kernel<T>;
    if (smem > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return e;
    }
    return launch_kernel(kern, dim3((tokens + 63) / 64, kv_heads), dim3(kThreads), smem, (cudaStream_t)stream, pdl != 0, a);
  });
}

// Means of the blocks of `pool` tokens (counted from the sequence's start) that the portions complete, from the cache's rows
// into its rows of blocks; kp / vt with pool_row (all null, or whole prompts): also [rows, ld_kp], [heads * vdim, ld_vt] from
// row pool_row[portion] on.  longest: tokens of the longest portion.
IPEX_API int ipex_kv_pool(const void* kc, int64_t k_slot, int64_t k_head, const void* vc, int64_t v_slot, int64_t v_head,
                          void* pk, int64_t pk_slot, int64_t pk_head, void* pv, int64_t pv_slot, int64_t pv_head, void* kp,
                          int64_t ld_kp, void* vt, int64_t ld_vt, const int* pool_row, const int* slot, const int* pos,
                          const int* start, const int* seq_row, const int* seq_len, int seqs, int longest, int kv_heads,
                          int dim, int vdim, int pool, int dtype, void* stream) {
  if (seqs < 1 || seqs > 65535 || longest < 1 || kv_heads < 1 || kv_heads > 65535 || dim < 1 || vdim < 1 || pool < 1 ||
      (kp == nullptr) != (vt == nullptr) || (kp == nullptr) != (pool_row == nullptr))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const PoolArgs a = {kc, vc, pk, pv, kp, vt, slot, pos, start, seq_row, seq_len, pool_row, k_slot, k_head, v_slot, v_head,
                        pk_slot, pk_head, pv_slot, pv_head, ld_kp, ld_vt, pool, dim, vdim};
    const int blocks = longest / pool + 1;           // that a portion can complete
    kv_pool_kernel<T><<<dim3((blocks + kThreads / 32 - 1) / (kThreads / 32), kv_heads, seqs), kThreads, 0, (cudaStream_t)stream>>>(a);
    return cudaGetLastError();
  });
}

// Queries and keys of many tokens in place, x [tokens, ld] with `heads` of `dim`: pairs (i, i + half) turn by the tables'
// angles for the token's place in its sequence; before that, unit: divided by sqrt(mean square + eps), and times wq (the
// first q_heads heads) or wk (the others), [dim] each, unless null.
IPEX_API int ipex_qk_prepare(void* x, int64_t ld, const int* slot, const int* pos, const int* start, const float* cosp,
                             const float* sinp, int half, int unit, float eps, const float* wq, const float* wk, int q_heads,
                             int tokens, int heads, int dim, int dtype, int pdl, void* stream) {
  if (tokens < 1 || heads < 1 || dim < 1 || half < 0 || 2 * half > dim || (half > 0 && (cosp == nullptr || sinp == nullptr)))
    return (int)cudaErrorInvalidValue;
  const int64_t rows = (int64_t)tokens * heads, blocks = (rows + kThreads / 32 - 1) / (kThreads / 32);
  if (blocks > 0x7fffffff) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const Prepare p = {cosp, sinp, half, unit, eps, wq, wk, q_heads};
    constexpr int VN = 16 / (int)sizeof(T);
    if (rows < (1u << 31) && dim % VN == 0 && dim / VN <= 32 && half % VN == 0 && ld % VN == 0 &&
        (((uintptr_t)x | (uintptr_t)cosp | (uintptr_t)sinp) & 15) == 0) {
      cudaStream_t st = (cudaStream_t)stream;
      if (dim / VN <= 8) return launch_prepare<T, 8>(x, ld, slot, pos, start, p, rows, heads, dim, pdl != 0, st);
      if (dim / VN <= 16) return launch_prepare<T, 16>(x, ld, slot, pos, start, p, rows, heads, dim, pdl != 0, st);
      return launch_prepare<T, 32>(x, ld, slot, pos, start, p, rows, heads, dim, pdl != 0, st);
    }
    return launch_kernel(qk_prepare_kernel<T>, dim3((unsigned)blocks), dim3(kThreads), 0, (cudaStream_t)stream, pdl != 0,
                         (T*)x, ld, slot, pos, start, p, rows, heads, dim);
  });
}

// Attention of `tokens` query tokens (q: rows of ldq elements, `heads` of `dim`) over positions
// [max(start, pos - window + 1), pos] of their slots (window 0: unlimited; chunk > 0: those of the query's own chunk, counted
// from start).  append: file the tokens' own rows k / v (same row stride as q, v mixed with vfirst) first - then no two
// tokens may share a slot; otherwise the cache holds them.  prepare (with append): queries and new keys are rotated and
// normed on the way (see ipex_qk_prepare).  pool > 0 (with a window): beside it, the blocks of `pool` tokens that lie wholly
// before it, from pk / pv; append files the block that a token completes.  nsplit: CTAs (1, 2, 4 or 8) the keys of a token are shared by.  sink: one more
// score without a value in every softmax, 0 or sinks[head].  gate (may be null): outputs times gate_scale * sigmoid.
IPEX_API int ipex_kv_attn(const void* q, const void* k, const void* v, int64_t ldq, const void* vfirst, int64_t ld_vf,
                          float lambda, void* kc, int64_t k_slot, int64_t k_head, void* vc, int64_t v_slot,
                          int64_t v_head, void* out, int64_t ldo, const int* slot, const int* pos, const int* start,
                          int tokens, int heads, int kv_heads, int dim, int vdim, int window, int chunk, int sink,
                          const float* sinks, const void* gate, int64_t ldg, float gate_scale, int append, int prepare,
                          const float* cosp, const float* sinp, int half, int unit, float eps, const float* wq,
                          const float* wk, int pool, void* pk, int64_t pk_slot, int64_t pk_head, void* pv, int64_t pv_slot,
                          int64_t pv_head, int nsplit, float scale, int dtype, int pdl, void* stream) {
  if (tokens < 1 || tokens > 65535 || kv_heads < 1 || heads % kv_heads != 0 || dim < 1 || vdim < 1 || window < 0 || chunk < 0 ||
      nsplit < 1 || nsplit > 8 || (nsplit & (nsplit - 1)))
    return (int)cudaErrorInvalidValue;
  if (pool < 0 || (pool > 0 && (window < 1 || chunk > 0 || pk == nullptr || pv == nullptr))) return (int)cudaErrorInvalidValue;
  if (prepare && (!append || half < 0 || 2 * half > dim || (half > 0 && (cosp == nullptr || sinp == nullptr))))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    constexpr int VN = 16 / (int)sizeof(T);
    AttnArgs a = {q, k, v, vfirst, kc, vc, out, slot, pos, start, ldq, ld_vf, ldo, k_slot, k_head, v_slot, v_head,
                  lambda, scale, heads, kv_heads, dim, vdim, window, sink, append, chunk, sinks, gate, ldg, gate_scale,
                  {cosp, sinp, half, unit, eps, wq, wk, heads}, prepare, pool, pk, pv, pk_slot, pk_head, pv_slot, pv_head};
    const bool vec = dim % VN == 0 && vdim % VN == 0 && vdim / VN <= kThreads &&
                     (((uintptr_t)kc | (uintptr_t)vc | (uintptr_t)pk | (uintptr_t)pv) & 15) == 0;
    cudaStream_t st = (cudaStream_t)stream;
    if (vec) return pick_rows<T, true>(a, tokens, nsplit, pdl != 0, st);
    if (vdim > kThreads) return cudaErrorInvalidValue;
    return pick_rows<T, false>(a, tokens, nsplit, pdl != 0, st);
  });
}
