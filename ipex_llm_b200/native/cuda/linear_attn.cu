// Gated linear attention with a decay per key channel, sm_100a.
//
// Per head a matrix state S [dim, vdim] is carried from token to token:
//     S <- diag(alpha) S + k v^T;   o = S^T q      alpha = sigmoid(z)^(1 / tau),  z = up . low + bias
// q (times dim^-1/2), k, v come from projections; z from a low-rank pair whose first half (`low`) is a projection too.
// z, alpha and everything behind them, the state and the products that touch it are fp32.
//
//   linear_step    token by token, state in registers: decoding (one token of every sequence; the gated norm of the output
//                  is fused), short portions, 32-bit models
//   linear_prep    prompts, first half, parallel over chunks of 32 tokens: the decayed queries Q[t] = q_t prod_{s<=t} alpha_s
//                  and keys K[i] = k_i prod_{s>i} alpha_s, the scores P[t,i] = q_t . (k_i prod_{i<s<=t} alpha_s), i <= t
//   linear_chunks  second half, sequential over a sequence's chunks: O = Q S + P V, S <- diag(prod alpha) S + K^T V
//
// The chunked form multiplies decays and never divides by them or takes differences of their logarithms: inside halves
// of 16 tokens the scores run the product along, between the halves both factors are products that end or start at the
// border, so nothing overflows and nothing cancels however fast a channel forgets.  Products run on the tensor cores
// with fp32 operands split into tf32 pairs (values as they come from a 16-bit projection need one part only).  The state
// lives transposed in accumulator fragments, which serve as the left operand of the next chunk's read-out as they are.
//
// What lies before a sequence's first token counts as zero, so a slot needs no clearing when it changes hands.
#include <cooperative_groups.h>

#include "common/state_cols.cuh"
#include "common/tf32_pairs.cuh"
#include "common/utils.cuh"
#include "tcgen05_common.cuh"

namespace {

namespace cg = cooperative_groups;

constexpr int kThreads = 256;
constexpr int kC = 32;                // tokens per chunk
constexpr int kVS = 32;               // state columns per CTA of the chunked form
constexpr size_t kSmemMax = 226 * 1024;

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

struct Common {
  const void* proj;       // T [tokens, ldp]: q heads, k heads, v heads, output gates
  const float* low;       // [tokens, rank]
  const void* up;         // T [heads * dim, rank]
  const float* bias;      // [heads * dim]
  float* state;           // [slots, heads, dim, vdim]
  const int* slot;        // [tokens]
  const int* pos;         // [tokens]
  const int* start;       // [slots]
  const int* seq_row;     // [sequences] first packed token, or null: sequence = token
  const int* seq_len;
  int64_t ldp;
  int heads, dim, vdim, rank;
  float qscale, inv_tau;
};

__device__ __forceinline__ float channel_decay(float z, float inv_tau) {
  const float log_sigmoid = fminf(z, 0.f) - logf(1.0f + expf(-fabsf(z)));    // the sum's rounding is an error of 2^-24 here
  return expf(log_sigmoid * inv_tau);
}

// ---------------------------------------------------------------------------------------------- token by token
struct StepArgs {
  Common c;
  const void* norm_w;     // fused norm (one token per sequence): T [vdim], out T [tokens, ldo]
  void* out;
  float* raw;             // else: o [tokens, heads, vdim]
  int64_t ldo;
  float eps, out_scale;
  int gate_off;           // column of the output gates in proj
  int prefetch;           // slots are final before the kernels in front of this one end: fetch states early
  int staged;             // the head's rows of `up` fit shared memory
};

// A warp owns the state rows warp, warp + 8, ...; a lane CV neighbouring columns of the CTA's 32 CV.
template <typename T, int NR, int CV>
__global__ void __launch_bounds__(kThreads, NR <= 16 ? 2 : 1) linear_step_kernel(StepArgs s) {
  constexpr int VS = 32 * CV;
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, sq_id = blockIdx.z, slice = blockIdx.x;
  const int v0 = slice * VS, nv = min(VS, V - v0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c0 = lane * CV;
  const int ldb = 3 * D + VS, ldr = a.rank | 1;
  float* red = sm;                      // [2][8][VS]
  float* buf = red + 2 * 8 * VS;        // [2][3 D + VS]: q, k, alpha, v of a token
  float* sup = buf + 2 * ldb;           // [D][rank | 1]
  __shared__ float s_ss;
  const int row0 = a.seq_row != nullptr ? a.seq_row[sq_id] : sq_id, len = a.seq_len != nullptr ? a.seq_len[sq_id] : 1;
  const int qc = h * D, kc = a.heads * D + h * D, vc = 2 * a.heads * D + h * V + v0;
  const bool col = c0 < nv;             // CV divides V: a lane's columns exist together
  pdl_launch_dependents();
  if (s.prefetch) {
    // slots do not change while a step is in flight; the state's rows come to L2 while the projections finish
    const float* st = a.state + (((int64_t)a.slot[row0] * a.heads + h) * D) * V + v0;
    if (nv == V) {
      if (tid == 0) prefetch_l2_bulk(st, (uint32_t)(D * V * sizeof(float)));
    } else {
      for (int d = tid; d < D; d += kThreads) prefetch_l2_bulk(st + (int64_t)d * V, (uint32_t)(nv * sizeof(float)));
    }
  }
  const T* up = reinterpret_cast<const T*>(a.up) + (int64_t)h * D * a.rank;
  const float* bias = a.bias + h * D;
  if (s.staged)
    for (int i = tid; i < D * a.rank; i += kThreads) sup[i / a.rank * ldr + i % a.rank] = DT<T>::to_f(up[i]);
  float nw[CV];
#pragma unroll
  for (int c = 0; c < CV; ++c)
    nw[c] = s.raw == nullptr && col ? DT<T>::to_f(reinterpret_cast<const T*>(s.norm_w)[v0 + c0 + c]) : 0.f;
  if (s.staged) __syncthreads();
  pdl_wait();
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0 + c0;
  float S[NR][CV];
  const bool fresh = p0 <= start;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = warp + 8 * i;
#pragma unroll
    for (int c = 0; c < CV; ++c) S[i][c] = 0.f;
    if (col && d < D) load_cols<CV>(st + (int64_t)d * V, S[i]);
  }
  if (fresh) {
#pragma unroll
    for (int i = 0; i < NR; ++i)
#pragma unroll
      for (int c = 0; c < CV; ++c) S[i][c] = 0.f;
  }
  auto fetch = [&](int j) {             // token j of the sequence into its buffer
    const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)(row0 + j) * a.ldp;
    const float* low = a.low + (int64_t)(row0 + j) * a.rank;
    float* q = buf + (j & 1) * ldb;
    for (int i = tid; i < 3 * D + nv; i += kThreads) {
      float x;
      if (i < D) {
        // the decays first: theirs is the longest chain
        const T* u = up + (int64_t)i * a.rank;
        const float* su = sup + i * ldr;
        float z0 = bias[i], z1 = 0.f;
        int r = 0;
        for (; r + 1 < a.rank; r += 2) {
          z0 = fmaf(low[r], s.staged ? su[r] : DT<T>::to_f(u[r]), z0);
          z1 = fmaf(low[r + 1], s.staged ? su[r + 1] : DT<T>::to_f(u[r + 1]), z1);
        }
        if (r < a.rank) z0 = fmaf(low[r], s.staged ? su[r] : DT<T>::to_f(u[r]), z0);
        q[2 * D + i] = channel_decay(z0 + z1, a.inv_tau);
      } else if (i < 2 * D) {
        x = DT<T>::to_f(proj[qc + i - D]);
        q[i - D] = x * a.qscale;
      } else if (i < 3 * D) {
        x = DT<T>::to_f(proj[kc + i - 2 * D]);
        q[i - D] = x;
      } else {
        q[i] = DT<T>::to_f(proj[vc + i - 3 * D]);
      }
    }
  };
  float gate[CV];
  if (s.raw == nullptr && warp == 0 && col) {
#pragma unroll
    for (int c = 0; c < CV; ++c)
      gate[c] = DT<T>::to_f(reinterpret_cast<const T*>(a.proj)[(int64_t)row0 * a.ldp + s.gate_off + h * V + v0 + c0 + c]);
  }
  fetch(0);
  __syncthreads();
  for (int j = 0; j < len; ++j) {
    const float* q = buf + (j & 1) * ldb;
    float* rd = red + (j & 1) * (8 * VS);
    float v[CV], o[CV];
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      o[c] = 0.f;
      v[c] = col ? q[3 * D + c0 + c] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float qd = q[d], kd = q[D + d], ad = q[2 * D + d];
#pragma unroll
        for (int c = 0; c < CV; ++c) {
          S[i][c] = fmaf(kd, v[c], ad * S[i][c]);
          o[c] = fmaf(S[i][c], qd, o[c]);
        }
      }
    }
    store_cols<CV>(rd + warp * VS + c0, o);
    if (j + 1 < len) fetch(j + 1);
    __syncthreads();
    if (warp != (j & 7)) continue;      // the warps take turns with the sums
#pragma unroll
    for (int c = 0; c < CV; ++c) o[c] = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      float x[CV];
      load_cols<CV>(rd + w * VS + c0, x);
#pragma unroll
      for (int c = 0; c < CV; ++c) o[c] += x[c];
    }
    if (s.raw != nullptr && col) {
#pragma unroll
      for (int c = 0; c < CV; ++c) s.raw[((int64_t)(row0 + j) * a.heads + h) * V + v0 + c0 + c] = o[c];
    }
    if (s.raw == nullptr) {             // one token: warp 0 finishes it below
#pragma unroll
      for (int c = 0; c < CV; ++c) rd[c0 + c] = o[c];
    }
  }
  if (s.raw == nullptr) {
    // norm over all columns of the head, which the CTAs of the cluster hold slice by slice
    float o[CV], ss = 0.f;
    if (warp == 0) {
#pragma unroll
      for (int c = 0; c < CV; ++c) {
        o[c] = col ? red[c0 + c] : 0.f;
        ss = fmaf(o[c], o[c], ss);
      }
    }
    float total = ss = warp_sum(ss);
    if (gridDim.x > 1) {
      if (tid == 0) s_ss = ss;
      cg::cluster_group cluster = cg::this_cluster();
      cluster.sync();
      total = 0.f;
      for (int r = 0; r < (int)gridDim.x; ++r) total += *cluster.map_shared_rank(&s_ss, r);
      cluster.sync();
    }
    if (warp == 0 && col) {
      const float inv = s.out_scale / sqrtf(total / (float)V + s.eps);
      T* out = reinterpret_cast<T*>(s.out) + (int64_t)row0 * s.ldo + h * V + v0 + c0;
#pragma unroll
      for (int c = 0; c < CV; ++c) out[c] = DT<T>::from_f(o[c] * inv * nw[c] * silu(gate[c]));
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = warp + 8 * i;
    if (col && d < D) store_cols<CV>(st + (int64_t)d * V, S[i]);
  }
}

// ---------------------------------------------------------------------------------------------- in chunks
// Scratch of one (chunk, head), laid out like the shared memory that reads it (row strides keep the fragments' banks
// apart): Q and K of 32 rows, P [32][36], decay of the whole chunk per channel; then V [32][40] per slice of 32 columns.
struct Scratch {
  static constexpr int ldp = 36, ldv = 40;
  int Dp, slices, ld;
  __host__ __device__ Scratch(int D, int V)
      : Dp((D + 7) / 8 * 8), slices((V + kVS - 1) / kVS), ld(Dp % 16 == 0 ? Dp + 8 : Dp) {}
  __host__ __device__ int k() const { return kC * ld; }
  __host__ __device__ int p() const { return 2 * kC * ld; }
  __host__ __device__ int g() const { return p() + kC * ldp; }
  __host__ __device__ int shared_part() const { return g() + Dp; }
  __host__ __device__ int v(int slice) const { return shared_part() + slice * kC * ldv; }
  __host__ __device__ int floats() const { return v(slices); }
  __host__ __device__ int stage() const { return shared_part() + kC * ldv; }
};

struct ChunkArgs {
  Common c;
  const int* chunk_seq;     // [all chunks] sequence of a chunk
  const int* seq_chunk;     // [sequences + 1] first chunk of a sequence
  float* scratch;           // of the chunks [c0, c1), [chunk - c0][head]
  float* raw;               // o [tokens, heads, vdim]
  int* err;
  int c0, c1;
};

constexpr int kLdPart = 17;
size_t prep_smem(const Scratch& L, int rank) {
  return ((size_t)3 * kC * L.ld + (size_t)kC * rank + (size_t)rank * (L.Dp + 1) + 4 * 16 * kLdPart) * sizeof(float);
}

template <typename T>
__global__ void __launch_bounds__(kThreads) linear_prep_kernel(ChunkArgs s) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, chunk = s.c0 + blockIdx.x, rank = a.rank;
  const Scratch L(D, V);
  const int Dp = L.Dp, ld = L.ld;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* sq = sm;                        // [32][ld]
  float* sk = sq + kC * ld;
  float* sa = sk + kC * ld;              // decays
  float* part = sa + kC * ld;            // [4][16][17]
  float* slow = part + 4 * 16 * kLdPart; // [32][rank]
  float* sup = slow + kC * rank;         // [rank][Dp + 1]
  const int seq = s.chunk_seq[chunk], row0 = a.seq_row[seq], off = (chunk - s.seq_chunk[seq]) * kC;
  const int n = min(kC, a.seq_len[seq] - off), t0 = row0 + off;
  float* out = s.scratch + ((int64_t)(chunk - s.c0) * a.heads + h) * L.floats();
  const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)t0 * a.ldp;

  // ---- operands (zeros behind the sequence's end and past the sizes)
  const T* up = reinterpret_cast<const T*>(a.up) + (int64_t)h * D * rank;
  for (int i = tid; i < D * rank; i += kThreads) sup[i % rank * (Dp + 1) + i / rank] = DT<T>::to_f(up[i]);
  for (int i = tid; i < kC * rank; i += kThreads) slow[i] = i / rank < n ? a.low[(int64_t)t0 * rank + i] : 0.f;
  const int qc = h * D, kcol = a.heads * D + h * D, vcol = 2 * a.heads * D + h * V, Vp = L.slices * kVS;
  const bool vec = D % 8 == 0 && V % 8 == 0 && a.ldp % 8 == 0 && (reinterpret_cast<uintptr_t>(a.proj) & 15) == 0;
  if (vec) {
    const int nd = D / 8, nvv = Vp / 8, per = 2 * nd + nvv;
    for (int i = tid; i < kC * per; i += kThreads) {
      const int t = i / per, c = i % per;
      const int what = c < nd ? 0 : c < 2 * nd ? 1 : 2, e0 = (what == 0 ? c : what == 1 ? c - nd : c - 2 * nd) * 8;
      uint4 raw = make_uint4(0, 0, 0, 0);
      if (t < n && (what < 2 || e0 < V))
        raw = *reinterpret_cast<const uint4*>(proj + (int64_t)t * a.ldp + (what == 0 ? qc : what == 1 ? kcol : vcol) + e0);
      const T* e = reinterpret_cast<const T*>(&raw);
      const float f = what == 0 ? a.qscale : 1.f;
      float* dst = what == 0 ? sq + t * ld + e0 : what == 1 ? sk + t * ld + e0
                                                            : out + L.v(e0 / kVS) + t * L.ldv + e0 % kVS;
#pragma unroll
      for (int j = 0; j < 8; j += 4)
        *reinterpret_cast<float4*>(dst + j) = make_float4(DT<T>::to_f(e[j]) * f, DT<T>::to_f(e[j + 1]) * f,
                                                          DT<T>::to_f(e[j + 2]) * f, DT<T>::to_f(e[j + 3]) * f);
    }
  } else {
    for (int i = tid; i < kC * Dp; i += kThreads) {
      const int t = i / Dp, d = i % Dp;
      const bool on = t < n && d < D;
      sq[t * ld + d] = on ? DT<T>::to_f(proj[(int64_t)t * a.ldp + qc + d]) * a.qscale : 0.f;
      sk[t * ld + d] = on ? DT<T>::to_f(proj[(int64_t)t * a.ldp + kcol + d]) : 0.f;
    }
    for (int i = tid; i < kC * Vp; i += kThreads) {
      const int t = i / Vp, c = i % Vp;
      out[L.v(c / kVS) + t * L.ldv + c % kVS] = t < n && c < V ? DT<T>::to_f(proj[(int64_t)t * a.ldp + vcol + c]) : 0.f;
    }
  }
  __syncthreads();
  // ---- decays: eight tokens of a channel per item
  for (int i = tid; i < Dp * (kC / 8); i += kThreads) {
    const int d = i % Dp, tb = i / Dp * 8;
    float z[8];
    const float b = d < D ? a.bias[h * D + d] : 0.f;
#pragma unroll
    for (int t = 0; t < 8; ++t) z[t] = b;
    if (d < D)
      for (int r = 0; r < rank; ++r) {
        const float u = sup[r * (Dp + 1) + d];
#pragma unroll
        for (int t = 0; t < 8; ++t) z[t] = fmaf(slow[(tb + t) * rank + r], u, z[t]);
      }
#pragma unroll
    for (int t = 0; t < 8; ++t) sa[(tb + t) * ld + d] = tb + t < n && d < D ? channel_decay(z[t], a.inv_tau) : 1.f;
  }
  __syncthreads();
  // ---- scores inside the two halves of 16 tokens: a unit of eight lanes takes key i, a lane every eighth channel
  {
    const int half = warp >> 2, u0 = (warp & 3) * 4, i = u0 + (lane >> 3), base = half * 16;
    float acc[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) acc[t] = 0.f;
    for (int d = lane & 7; d < Dp; d += 8) {
      float w = sk[(base + i) * ld + d];
      const float* qd = sq + base * ld + d;
      const float* ad = sa + base * ld + d;
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        if (t >= u0) {                       // the same for the whole warp
          if (t > i) w *= ad[t * ld];
          if (t >= i) acc[t] = fmaf(qd[t * ld], w, acc[t]);
        }
      }
    }
    fold<16, 4>(acc, lane);                  // a lane keeps two neighbouring tokens
    const int first = ((lane & 4) ? 8 : 0) + ((lane & 2) ? 4 : 0) + ((lane & 1) ? 2 : 0);
    float* P = out + L.p();
#pragma unroll
    for (int j = 0; j < 2; ++j) P[(base + first + j) * L.ldp + base + i] = acc[j];
    if (half == 0)                           // keys of the second half are not seen by the first
#pragma unroll
      for (int j = 0; j < 2; ++j) P[(first + j) * L.ldp + 16 + i] = 0.f;
  }
  __syncthreads();
  // ---- decayed queries and keys; what meets between the halves stays in shared memory
  for (int i = tid; i < 2 * Dp; i += kThreads) {
    const int d = i % Dp;
    const float* ad = sa + d;
    if (i < Dp) {
      float run = 1.f, all;
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        run *= ad[t * ld];
        out[t * ld + d] = sq[t * ld + d] * run;
      }
      all = run;
      run = 1.f;
#pragma unroll
      for (int t = 16; t < 32; ++t) {
        run *= ad[t * ld];
        const float x = sq[t * ld + d] * run;
        sq[t * ld + d] = x;
        out[t * ld + d] = x * all;
      }
      out[L.g() + d] = all * run;
    } else {
      float* kd = out + L.k() + d;
      float run = 1.f, all;
#pragma unroll
      for (int t = 31; t >= 16; --t) {
        kd[t * ld] = sk[t * ld + d] * run;
        run *= ad[t * ld];
      }
      all = run;
      run = 1.f;
#pragma unroll
      for (int t = 15; t >= 0; --t) {
        const float x = sk[t * ld + d] * run;
        sk[t * ld + d] = x;
        kd[t * ld] = x * all;
        run *= ad[t * ld];
      }
    }
  }
  __syncthreads();
  // ---- scores of the second half's queries with the first half's keys: two column tiles, four shares of the channels
  {
    const int n0 = (warp & 1) * 8, share = warp >> 1, steps = Dp / 8;
    float c[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = share; k < steps; k += 4)
      mac3(c, frag_a([&](int r, int kk) { return sq[(16 + r) * ld + k * 8 + kk]; }, g, t4),
           frag_b([&](int kk, int j) { return sk[(n0 + j) * ld + k * 8 + kk]; }, g, t4));
#pragma unroll
    for (int i = 0; i < 4; ++i) part[(share * 16 + g + 8 * (i >> 1)) * kLdPart + n0 + 2 * t4 + (i & 1)] = c[i];
  }
  __syncthreads();
  {
    const int t = tid >> 4, i = tid & 15;
    float x = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) x += part[(k * 16 + t) * kLdPart + i];
    out[L.p() + (16 + t) * L.ldp + i] = x;
  }
}

size_t chunk_smem(const Scratch& L, int stages) {
  return ((size_t)stages * L.stage() + 2 * 4 * kC * 36) * sizeof(float);
}

// CTA = 32 state columns of one head of one sequence.  Warp (vt, dg): columns 16 vt .. + 15, channel tiles of share dg; S^T
// in accumulator fragments.  The four shares' read-outs meet in shared memory.
template <typename T, int MT>
__global__ void __launch_bounds__(kThreads, 1) linear_chunks_kernel(ChunkArgs s, int stages) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(8) uint64_t full[4];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kVS, nv = min(kVS, V - v0);
  const Scratch L(D, V);
  const int Dp = L.Dp, ld = L.ld, tiles = Dp / 8, per = (tiles + 3) / 4;
  const int first = s.seq_chunk[seq], last = s.seq_chunk[seq + 1];
  const int ca = max(first, s.c0), cb = min(last, s.c1);
  if (ca >= cb) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int vt = warp & 1, dg = warp >> 1;
  float* red = sm + stages * L.stage();        // [2][4][32][36]
  const int row0 = a.seq_row[seq], len = a.seq_len[seq];
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0;
  auto fetch = [&](int c) {                    // one thread
    if (c >= cb) return;
    const float* src = s.scratch + ((int64_t)(c - s.c0) * a.heads + h) * L.floats();
    float* dst = sm + ((c - ca) % stages) * L.stage();
    uint64_t* bar = &full[(c - ca) % stages];
    tc5::mbar_expect_tx(bar, (uint32_t)(L.stage() * sizeof(float)));
    bulk_load(dst, src, (uint32_t)(L.shared_part() * sizeof(float)), bar);
    bulk_load(dst + L.shared_part(), src + L.v(blockIdx.x), (uint32_t)(kC * L.ldv * sizeof(float)), bar);
  };
  if (tid == 0) {
    for (int i = 0; i < 4; ++i) tc5::mbar_init(&full[i], 1);
    abort_word = 0;
    tc5::fence_barrier_init();
    for (int i = 0; i < stages; ++i) fetch(ca + i);
  }
  const bool fresh = ca == first && p0 <= start;
  float S[MT][4];                              // columns g, g + 8 of the warp's 16; channels 2 t, 2 t + 1 of a tile
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int tile = dg * per + m, d = tile * 8 + 2 * t4 + (i & 1), c = vt * 16 + g + 8 * (i >> 1);
      S[m][i] = m < per && !fresh && d < D && c < nv ? st[(int64_t)d * V + c] : 0.f;
    }
  __syncthreads();
  bool ok = true;
  for (int c = ca; c < cb; ++c) {
    const int at = c - ca;
    if (!tc5::mbar_wait(&full[at % stages], (at / stages) & 1, abort_flag)) {
      if (lane == 0) tc5::report(s.err, 41);
      ok = false;
    }
    if (ok) {
      const float* Q = sm + (at % stages) * L.stage();
      const float *K = Q + L.k(), *P = Q + L.p(), *G = Q + L.g(), *Vs = Q + L.shared_part() + vt * 16;
      // ---- O^T = S^T Q^T: the state's fragments are the left operand (k order inside a tile: 0 2 4 6 1 3 5 7)
      float o[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int tile = dg * per + m;
        if (m < per && tile < tiles) {
          FragA fa;
          split_tf32(S[m][0], fa.hi[0], fa.lo[0]);
          split_tf32(S[m][2], fa.hi[1], fa.lo[1]);
          split_tf32(S[m][1], fa.hi[2], fa.lo[2]);
          split_tf32(S[m][3], fa.hi[3], fa.lo[3]);
          FragB fb[4];
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            const float2 q = *reinterpret_cast<const float2*>(Q + (n * 8 + g) * ld + tile * 8 + 2 * t4);
            split_tf32(q.x, fb[n].hi[0], fb[n].lo[0]);
            split_tf32(q.y, fb[n].hi[1], fb[n].lo[1]);
          }
          // four independent chains side by side
#pragma unroll
          for (int n = 0; n < 4; ++n) mma_tf32(o[n], fa.lo, fb[n].hi);
#pragma unroll
          for (int n = 0; n < 4; ++n) mma_tf32(o[n], fa.hi, fb[n].lo);
#pragma unroll
          for (int n = 0; n < 4; ++n) mma_tf32(o[n], fa.hi, fb[n].hi);
        }
      }
      // values as left operands, exact in one part
      uint32_t va[4][4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float* v = Vs + (k * 8 + t4) * L.ldv + g;
        va[k][0] = __float_as_uint(v[0]);
        va[k][1] = __float_as_uint(v[8]);
        va[k][2] = __float_as_uint(v[4 * L.ldv]);
        va[k][3] = __float_as_uint(v[4 * L.ldv + 8]);
      }
      // ---- ... + V^T P^T, this warp's eight keys
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (k == dg) {
#pragma unroll
          for (int n = 0; n < 4; ++n)
            if (n >= k) mac2(o[n], va[k], frag_b([&](int kk, int j) { return P[(n * 8 + j) * L.ldp + k * 8 + kk]; }, g, t4));
        }
      float* rd = red + ((at & 1) * 4 + dg) * (kC * 36) + vt * 16;
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) rd[(n * 8 + 2 * t4 + (i & 1)) * 36 + g + 8 * (i >> 1)] = o[n][i];
      // ---- S^T <- S^T diag(G) + V^T K
      const int mine = min(per, tiles - dg * per);       // tiles of this warp that exist
      float add[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i) add[m][i] = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        FragB fb[MT];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < mine)
            fb[m] = frag_b([&](int kk, int j) { return K[(k * 8 + kk) * ld + (dg * per + m) * 8 + j]; }, g, t4);
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < mine) mma_tf32(add[m], va[k], fb[m].lo);
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < mine) mma_tf32(add[m], va[k], fb[m].hi);
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
        if (m < mine) {
          const float2 gd = *reinterpret_cast<const float2*>(G + (dg * per + m) * 8 + 2 * t4);
          S[m][0] = fmaf(gd.x, S[m][0], add[m][0]);
          S[m][1] = fmaf(gd.y, S[m][1], add[m][1]);
          S[m][2] = fmaf(gd.x, S[m][2], add[m][2]);
          S[m][3] = fmaf(gd.y, S[m][3], add[m][3]);
        }
    }
    if (__syncthreads_or(!ok)) {               // the parts are in place, the stage is free again
      ok = false;
      break;
    }
    if (tid == 0) fetch(c + stages);
    const int off = (c - first) * kC;
    const float* rd = red + (at & 1) * 4 * (kC * 36);
#pragma unroll
    for (int i = 0; i < kC * kVS / kThreads; ++i) {
      const int t = warp + 8 * i;
      const float x = (rd[t * 36 + lane] + rd[(kC + t) * 36 + lane]) +
                      (rd[(2 * kC + t) * 36 + lane] + rd[(3 * kC + t) * 36 + lane]);
      if (off + t < len && lane < nv) s.raw[((int64_t)(row0 + off + t) * a.heads + h) * V + v0 + lane] = x;
    }
  }
  if (!ok) {                                   // copies in flight still write to this CTA's memory
    if (tid == 0)
      for (int i = 0; i < stages; ++i) {
        tc5::mbar_wait_quiet(&full[i], 0, 1 << 12);
        tc5::mbar_wait_quiet(&full[i], 1, 1 << 12);
      }
    return;
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int tile = dg * per + m, d = tile * 8 + 2 * t4 + (i & 1), c = vt * 16 + g + 8 * (i >> 1);
      if (m < per && d < D && c < nv) st[(int64_t)d * V + c] = S[m][i];
    }
}

bool sizes_ok(int heads, int dim, int vdim, int rank) {
  return heads >= 1 && heads <= 65535 && dim >= 1 && dim <= 512 && vdim >= 1 && vdim <= 65535 && rank >= 1;
}

template <typename T, int NR, int CV>
cudaError_t launch_step(StepArgs& s, int seqs, bool fused, bool pdl, cudaStream_t st) {
  const int slices = (s.c.vdim + 32 * CV - 1) / (32 * CV);
  if (fused && slices > 8) return cudaErrorInvalidValue;
  size_t smem = (2 * (3 * (size_t)s.c.dim + 32 * CV) + 2 * 8 * 32 * CV) * sizeof(float);
  const size_t up = (size_t)s.c.dim * (s.c.rank | 1) * sizeof(float);
  s.staged = smem + up <= 100 * 1024;
  if (s.staged) smem += up;
  if (smem > kSmemMax) return cudaErrorInvalidValue;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(linear_step_kernel<T, NR, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, s.c.heads, seqs);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (fused && slices > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = slices;
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
  return cudaLaunchKernelEx(&cfg, linear_step_kernel<T, NR, CV>, s);
}

// Columns per lane: as many as V divides into and the registers of NR rows leave room for, fewer while that spreads the
// large states of a few sequences over more SMs.
template <typename T, int NR>
cudaError_t pick_cols(StepArgs& s, int seqs, bool fused, bool pdl, cudaStream_t st) {
  const int V = s.c.vdim;
  int cv = NR <= 16 && V % 4 == 0 && V > 64 ? 4 : NR <= 32 && V % 2 == 0 && V > 32 ? 2 : 1;
  while (cv > 1 && s.c.dim * 32 * cv > 4096 && (int64_t)s.c.heads * seqs * ((V + 16 * cv - 1) / (16 * cv)) <= 2 * 148) cv /= 2;
  if constexpr (NR <= 16)
    if (cv == 4) return launch_step<T, NR, 4>(s, seqs, fused, pdl, st);
  if constexpr (NR <= 32)
    if (cv == 2) return launch_step<T, NR, 2>(s, seqs, fused, pdl, st);
  return launch_step<T, NR, 1>(s, seqs, fused, pdl, st);
}

Common common_args(const void* proj, int64_t ldp, const float* low, const void* up, const float* bias, float* state,
                   const int* slot, const int* pos, const int* start, const int* seq_row, const int* seq_len, int heads,
                   int dim, int vdim, int rank, float tau) {
  Common c = {proj, low, up, bias, state, slot, pos, start, seq_row, seq_len, ldp, heads, dim, vdim, rank,
              1.0f / sqrtf((float)dim), 1.0f / tau};
  return c;
}

}  // namespace

// Can the chunked form take these sizes?
IPEX_API int ipex_linear_chunks_ok(int dim, int vdim, int rank) {
  const Scratch L(dim, vdim);
  return dim >= 1 && dim <= 256 && vdim >= 1 && rank >= 1 && prep_smem(L, rank) <= kSmemMax && chunk_smem(L, 1) <= kSmemMax;
}
IPEX_API int64_t ipex_linear_scratch_floats(int dim, int vdim) { return Scratch(dim, vdim).floats(); }
// Can a decode step of these sizes norm its outputs on the way?
IPEX_API int ipex_linear_fused_ok(int vdim) { return vdim >= 1 && vdim <= 256; }

// Token by token.  seq_row / seq_len null: `seqs` sequences of one token each; norm_w / out [tokens, ldo] then take
// out_scale * norm(o) * norm_w * silu(gate) (vdim <= 256).  raw (when out is null): the plain outputs [tokens, heads, vdim].
IPEX_API int ipex_linear_step(const void* proj, int64_t ldp, int gate_off, const float* low, const void* up,
                              const float* bias, float* state, const int* slot, const int* pos, const int* start,
                              const int* seq_row, const int* seq_len, int seqs, const void* norm_w, float eps,
                              float out_scale, void* out, int64_t ldo, float* raw, int heads, int dim, int vdim, int rank,
                              float tau, int dtype, int pdl, void* stream) {
  if (!sizes_ok(heads, dim, vdim, rank) || seqs < 1 || seqs > 65535 || (seq_row == nullptr) != (seq_len == nullptr))
    return (int)cudaErrorInvalidValue;
  const bool fused = raw == nullptr;
  if (fused && (seq_row != nullptr || out == nullptr || norm_w == nullptr || !ipex_linear_fused_ok(vdim)))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    StepArgs s = {common_args(proj, ldp, low, up, bias, state, slot, pos, start, seq_row, seq_len, heads, dim, vdim, rank, tau),
                  norm_w, out, raw, ldo, eps, out_scale, gate_off, pdl && fused && vdim % 4 == 0, 0};
    cudaStream_t st = (cudaStream_t)stream;
    if (dim <= 32) return pick_cols<T, 4>(s, seqs, fused, pdl != 0, st);
    if (dim <= 64) return pick_cols<T, 8>(s, seqs, fused, pdl != 0, st);
    if (dim <= 128) return pick_cols<T, 16>(s, seqs, fused, pdl != 0, st);
    if (dim <= 256) return pick_cols<T, 32>(s, seqs, fused, pdl != 0, st);
    return pick_cols<T, 64>(s, seqs, fused, pdl != 0, st);
  });
}

// Chunks [c0, c1) of a packed batch in the chunked form (16-bit models).  chunk_seq [chunks], seq_chunk [seqs + 1]: device
// tables of the sequences' chunks of 32 tokens, in order; scratch: (c1 - c0) * heads * ipex_linear_scratch_floats; raw as
// above.
IPEX_API int ipex_linear_chunks(const void* proj, int64_t ldp, const float* low, const void* up, const float* bias,
                                float* state, const int* slot, const int* pos, const int* start, const int* seq_row,
                                const int* seq_len, int seqs, const int* chunk_seq, const int* seq_chunk, int c0, int c1,
                                float* scratch, float* raw, int heads, int dim, int vdim, int rank, float tau, int dtype,
                                int* err, void* stream) {
  if (!sizes_ok(heads, dim, vdim, rank) || !ipex_linear_chunks_ok(dim, vdim, rank) || seqs < 1 || seqs > 65535 || c0 < 0 ||
      c1 <= c0 || seq_row == nullptr || seq_len == nullptr || (((uintptr_t)scratch) & 15) || dtype == DT_F32)
    return (int)cudaErrorInvalidValue;
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ChunkArgs s = {common_args(proj, ldp, low, up, bias, state, slot, pos, start, seq_row, seq_len, heads, dim, vdim, rank, tau),
                   chunk_seq, seq_chunk, scratch, raw, err, c0, c1};
    cudaStream_t st = (cudaStream_t)stream;
    const Scratch L(dim, vdim);
    const size_t ps = prep_smem(L, rank);
    cudaError_t e = cudaFuncSetAttribute(linear_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ps);
    if (e != cudaSuccess) return e;
    linear_prep_kernel<T><<<dim3(c1 - c0, heads), kThreads, ps, st>>>(s);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    int stages = 4;
    while (stages > 1 && chunk_smem(L, stages) > kSmemMax) --stages;
    const size_t cs = chunk_smem(L, stages);
    auto kern = dim <= 64 ? linear_chunks_kernel<T, 2> : dim <= 128 ? linear_chunks_kernel<T, 4> : linear_chunks_kernel<T, 8>;
    e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cs);
    if (e != cudaSuccess) return e;
    kern<<<dim3(L.slices, heads, seqs), kThreads, cs, st>>>(s, stages);
    return cudaGetLastError();
  };
  return (int)(dtype == DT_F16 ? run((__half*)nullptr) : run((__nv_bfloat16*)nullptr));
}
