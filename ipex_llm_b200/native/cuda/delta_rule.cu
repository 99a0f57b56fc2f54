// Gated delta rule with short convolutions, sm_100a.
//
// Per head a matrix state S [dim, vdim] is carried from token to token:
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// q, k, v come from projections through a causal convolution over a few tokens (per channel) and silu; q and k are unit
// vectors.  State, gates, unit vectors and everything inside the recurrence are fp32.
//
//   delta_step    token by token, state in registers: decoding (one token of every sequence; the gated norm of the
//                 output is fused), short portions, 32-bit models
//   delta_prep    prompts, first half, parallel over chunks of 32 tokens: with L the running sum of log g inside a
//                 chunk and A[t,i] = beta_t e^(L_t - L_i) (k_t . k_i) for i < t, the chunk's updates solve
//                 (I + A) U = beta V - beta e^L K S, so  U = Ub - W S  with Ub = (I + A)^-1 beta V and
//                 W = (I + A)^-1 beta e^L K
//   delta_chunks  second half, sequential over a sequence's chunks: U = Ub - W S, O = e^L Q S + P U with
//                 P[t,i] = e^(L_t - L_i) (q_t . k_i) for i <= t, S <- e^L_end S + (e^(L_end - L) K)^T U
//
// The products of the chunked form run on the tensor cores with every fp32 operand split into two tf32 parts (three
// products, about 22 bits), accumulated in fp32; the state itself is only ever added to in fp32.  The state's columns
// are independent, so a head is spread over slices of 32 columns.
//
// Convolution inputs are kept in a ring of `taps` rows per slot (row = position mod taps): a decode step writes a row
// that no other block of the step reads.  What lies before a sequence's first token counts as zero, and so does the
// state there, so a slot needs no clearing when it changes hands.
#include <cooperative_groups.h>

#include "common/short_conv.cuh"
#include "common/state_cols.cuh"
#include "common/tf32_pairs.cuh"
#include "common/utils.cuh"
#include "tcgen05_common.cuh"

namespace {

namespace cg = cooperative_groups;

constexpr int kThreads = 256;
constexpr int kChunkThreads = 256;    // of the sequential half
constexpr int kC = 32;                // tokens per chunk
constexpr int kVS = 32;               // state columns per CTA of the chunked form

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

struct Common {
  const void* proj;       // T [tokens, ldp]: q heads, k heads, v heads, output gates
  const float* gates;     // [tokens, 2 heads]: write strengths, then decays, before their activations
  const void* conv;       // T [channels, taps] for the q, k and v channels
  const float* a_log;     // [heads]
  const float* dt_bias;   // [heads]
  void* ring;             // T [slots, taps, channels]
  float* state;           // [slots, heads, dim, vdim]
  const int* slot;        // [tokens]
  const int* pos;         // [tokens]
  const int* start;       // [slots]
  const int* seq_row;     // [sequences] first packed token, or null: sequence = token
  const int* seq_len;
  int64_t ldp;
  int heads, kv_heads, dim, vdim, taps, channels;
  float qscale;
};

constexpr float kUnitEps = 1e-6f;

// log of the decay and write strength of one token and head
__device__ __forceinline__ float log_decay(float a, float dt_bias, float a_log) {
  const float z = a + dt_bias;
  return -expf(a_log) * softplusf(z);
}

// ---------------------------------------------------------------------------------------------- token by token
struct StepArgs {
  Common c;
  const void* norm_w;     // fused norm (one token per sequence): T [vdim], out T [tokens, ldo]
  void* out;
  float* raw;             // else: o [tokens, heads, vdim]
  int64_t ldo;
  float eps;
  int gate_off;           // column of the output gates in proj
  int ring_write;         // one token per sequence: file its convolution inputs
  int prefetch;           // slots are final before the kernels in front of this one end: fetch states early
};

// A warp owns the state rows warp, warp + 8, ...; a lane CV neighbouring columns of the CTA's 32 CV.
template <typename T, int NR, int CV>
__global__ void __launch_bounds__(kThreads, NR * CV <= 64 ? 2 : 1) delta_step_kernel(StepArgs s) {
  constexpr int VS = 32 * CV;
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, sq_id = blockIdx.z, slice = blockIdx.x;
  const int hk = h / (a.heads / a.kv_heads), v0 = slice * VS, nv = min(VS, V - v0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c0 = lane * CV;
  float* red = sm;                      // [2][2][8][VS]
  float* buf = red + 2 * 2 * 8 * VS;    // [2][2 D + VS]: q, k, v of a token
  float* wt = buf + 2 * (2 * D + VS);   // [2 D + VS][taps]: convolution weights
  __shared__ float s_ss;
  const int row0 = a.seq_row != nullptr ? a.seq_row[sq_id] : sq_id, len = a.seq_len != nullptr ? a.seq_len[sq_id] : 1;
  const int qc = hk * D, kc = a.kv_heads * D + hk * D, vc = 2 * a.kv_heads * D + h * V + v0;
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
  for (int i = tid; i < 2 * D + nv; i += kThreads) {
    const int c = i < D ? qc + i : i < 2 * D ? kc + i - D : vc + i - 2 * D;
    for (int j = 0; j < a.taps; ++j) wt[i * a.taps + j] = DT<T>::to_f(reinterpret_cast<const T*>(a.conv)[(int64_t)c * a.taps + j]);
  }
  const float alog = a.a_log[h], dtb = a.dt_bias[h];
  float nw[CV];
#pragma unroll
  for (int c = 0; c < CV; ++c)
    nw[c] = s.raw == nullptr && col ? DT<T>::to_f(reinterpret_cast<const T*>(s.norm_w)[v0 + c0 + c]) : 0.f;
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
  for (int j = 0; j < len; ++j) {
    const int t = row0 + j, p = p0 + j;
    float* q = buf + (j & 1) * (2 * D + VS);
    float* k = q + D;
    float* v = k + D;
    float* rd = red + (j & 1) * (2 * 8 * VS);
    const float bg = a.gates[(int64_t)t * 2 * a.heads + h], ag = a.gates[(int64_t)t * 2 * a.heads + a.heads + h];
    float gate[CV];
    if (s.raw == nullptr && warp == 0 && col) {
#pragma unroll
      for (int c = 0; c < CV; ++c)
        gate[c] = DT<T>::to_f(reinterpret_cast<const T*>(a.proj)[(int64_t)t * a.ldp + s.gate_off + h * V + v0 + c0 + c]);
    }
    for (int i = tid; i < 2 * D + nv; i += kThreads) {
      const int c = i < D ? qc + i : i < 2 * D ? kc + i - D : vc + i - 2 * D;
      q[i] = conv_silu<T>(a, c, t, j, p, start, slot, wt + i * a.taps + a.taps - 1);
    }
    const float beta = sigmoidf(bg), g = expf(log_decay(ag, dtb, alog));
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int d = lane; d < D; d += 32) {
      qq = fmaf(q[d], q[d], qq);
      kk = fmaf(k[d], k[d], kk);
      qk = fmaf(q[d], k[d], qk);
    }
    float sk[CV], sq[CV];
#pragma unroll
    for (int c = 0; c < CV; ++c) sk[c] = sq[c] = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float kd = k[d], qd = q[d];
#pragma unroll
        for (int c = 0; c < CV; ++c) {
          sk[c] = fmaf(S[i][c], kd, sk[c]);
          sq[c] = fmaf(S[i][c], qd, sq[c]);
        }
      }
    }
    store_cols<CV>(rd + warp * VS + c0, sk);
    store_cols<CV>(rd + (8 + warp) * VS + c0, sq);
    const float iq = a.qscale / sqrtf(warp_sum(qq) + kUnitEps), ik = 1.0f / sqrtf(warp_sum(kk) + kUnitEps);
    qk = warp_sum(qk) * iq * ik;
    __syncthreads();
#pragma unroll
    for (int c = 0; c < CV; ++c) sk[c] = sq[c] = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      float x[CV], y[CV];
      load_cols<CV>(rd + w * VS + c0, x);
      load_cols<CV>(rd + (8 + w) * VS + c0, y);
#pragma unroll
      for (int c = 0; c < CV; ++c) {
        sk[c] += x[c];
        sq[c] += y[c];
      }
    }
    float u[CV], o[CV];
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      const float uc = col ? beta * (v[c0 + c] - g * ik * sk[c]) : 0.f;
      o[c] = g * iq * sq[c] + qk * uc;               // S^T q after the write
      u[c] = ik * uc;
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float kd = k[d];
#pragma unroll
        for (int c = 0; c < CV; ++c) S[i][c] = fmaf(kd, u[c], g * S[i][c]);
      }
    }
    if (s.raw != nullptr) {
      if (warp == 0 && col) {
#pragma unroll
        for (int c = 0; c < CV; ++c) s.raw[((int64_t)t * a.heads + h) * V + v0 + c0 + c] = o[c];
      }
    } else {
      // one token: norm over all columns of the head, which the CTAs of the cluster hold slice by slice
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < CV; ++c) ss = fmaf(o[c], o[c], ss);
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
        const float inv = 1.0f / sqrtf(total / (float)V + s.eps);
        T* out = reinterpret_cast<T*>(s.out) + (int64_t)t * s.ldo + h * V + v0 + c0;
#pragma unroll
        for (int c = 0; c < CV; ++c) out[c] = DT<T>::from_f(o[c] * inv * nw[c] * silu(gate[c]));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = warp + 8 * i;
    if (col && d < D) store_cols<CV>(st + (int64_t)d * V, S[i]);
  }
  if (s.ring_write) {
    // nobody reads this row in this launch; the first head of a group files the shared q / k channels
    T* ring = reinterpret_cast<T*>(a.ring) + ((int64_t)slot * a.taps + p0 % a.taps) * a.channels;
    const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)row0 * a.ldp;
    if (slice == 0 && h % (a.heads / a.kv_heads) == 0)
      for (int i = tid; i < 2 * D; i += kThreads) {
        const int c = i < D ? qc + i : kc + i - D;
        ring[c] = proj[c];
      }
    for (int i = tid; i < nv; i += kThreads) ring[vc + i] = proj[vc + i];
  }
}

// Scratch of one (chunk, head), laid out like the shared memory that reads it (row strides keep the fragments' banks
// apart): W, Q and K parts of 32 rows, P [32][36], decay of the whole chunk; then Ub [32][40] per slice of 32 columns.
struct Scratch {
  static constexpr int ldp = 36, ldu = 40;
  int Dp, slices, ldw, ldk;
  __host__ __device__ Scratch(int D, int V)
      : Dp((D + 7) / 8 * 8), slices((V + kVS - 1) / kVS), ldw(Dp + 4), ldk(Dp + 8) {}
  __host__ __device__ int q() const { return kC * ldw; }
  __host__ __device__ int k() const { return kC * 2 * ldw; }
  __host__ __device__ int p() const { return k() + kC * ldk; }
  __host__ __device__ int g() const { return p() + kC * ldp; }
  __host__ __device__ int shared_part() const { return g() + 4; }
  __host__ __device__ int ub(int slice) const { return shared_part() + slice * kC * ldu; }
  __host__ __device__ int floats() const { return ub(slices); }
  __host__ __device__ int stage() const { return shared_part() + kC * ldu; }
};

struct ChunkArgs {
  Common c;
  const int* chunk_seq;     // [all chunks] sequence of a chunk
  const int* seq_chunk;     // [sequences + 1] first chunk of a sequence
  float* scratch;           // of the chunks [c0, c1), [chunk - c0][head]
  float* raw;               // o [tokens, heads, vdim]
  int* err;
  int c0, c1;
  int vec;                  // rows of proj and ring can be read 16 bytes at a time
};

template <typename T, int TP>
__global__ void __launch_bounds__(kThreads, 3) delta_prep_kernel(ChunkArgs s) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, chunk = s.c0 + blockIdx.x;
  const Scratch L(D, V);
  const int Dp = L.Dp, Vp = L.slices * kVS, ldk = Dp + 4, ldv = Vp + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* sq = sm;                        // [32][Dp + 4]
  float* sk = sq + kC * ldk;             // [32][Dp + 4]
  float* sv = sk + kC * ldk;             // [32][Vp + 8]
  float* sA = sv + kC * ldv;             // [32][36]
  float* sT = sA + kC * 36;              // [32][36]
  // [32] running sum of log g, in 64-bit: its differences must keep 32-bit accuracy when single tokens decay to nothing
  double* sL = reinterpret_cast<double*>(sT + kC * 36);
  float* sB = reinterpret_cast<float*>(sL + kC);      // [32] beta
  float* sE = sB + kC;                                // [32] e^L
  const int seq = s.chunk_seq[chunk], hk = h / (a.heads / a.kv_heads);
  const int row0 = a.seq_row[seq], off = (chunk - s.seq_chunk[seq]) * kC, n = min(kC, a.seq_len[seq] - off);
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0] + off, t0 = row0 + off;
  float* out = s.scratch + ((int64_t)(chunk - s.c0) * a.heads + h) * L.floats();
  const int qc = hk * D, kcol = a.kv_heads * D + hk * D, vcol = 2 * a.kv_heads * D + h * V;

  // ---- convolutions (zeros behind the sequence's end and past the sizes)
  const T* taps_end = reinterpret_cast<const T*>(a.conv) + a.taps - 1;
  if (s.vec) {
    const int per = 2 * D + V, nvec = per / 8;
    float* ws = sA;                      // [taps][per], over what comes later (the launch checks that it fits)
    auto channel = [&](int c) { return c < D ? qc + c : c < 2 * D ? kcol + c - D : vcol + c - 2 * D; };
    for (int c = tid; c < per; c += kThreads) {
      const T* w = reinterpret_cast<const T*>(a.conv) + (int64_t)channel(c) * a.taps;
      for (int i = 0; i < a.taps; ++i) ws[i * per + c] = DT<T>::to_f(w[i]);
    }
    for (int i = tid; i < kC * (Vp - V); i += kThreads) sv[i / (Vp - V) * ldv + V + i % (Vp - V)] = 0.f;
    __syncthreads();
    for (int i = tid; i < nvec * (kC / 4); i += kThreads) {
      const int c = (i % nvec) * 8, first = (i / nvec) * 4;
      float acc[4][8];
      conv_block<T, TP>(a, channel(c), t0, row0, p0, start, slot, n, first, ws + c, per, acc);
      float* dst = c < D ? sq + c : c < 2 * D ? sk + c - D : sv + c - 2 * D;
      const int ld = c < 2 * D ? ldk : ldv;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const bool on = first + j < n;
#pragma unroll
        for (int e = 0; e < 8; e += 4)
          *reinterpret_cast<float4*>(dst + (first + j) * ld + e) =
              on ? make_float4(fast_silu(acc[j][e]), fast_silu(acc[j][e + 1]), fast_silu(acc[j][e + 2]),
                               fast_silu(acc[j][e + 3]))
                 : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    __syncthreads();                     // the weights' place is free
  } else {
    const int per = 2 * Dp + Vp;
    for (int i = tid; i < kC * per; i += kThreads) {
      const int t = i / per, c = i % per;
      float x = 0.f;
      if (c < 2 * Dp) {
        const int d = c < Dp ? c : c - Dp;
        if (t < n && d < D) {
          const int ch = (c < Dp ? qc : kcol) + d;
          x = conv_silu<T>(a, ch, t0 + t, off + t, p0 + t, start, slot, taps_end + (int64_t)ch * a.taps);
        }
        (c < Dp ? sq : sk)[t * ldk + d] = x;
      } else {
        const int d = c - 2 * Dp;
        if (t < n && d < V) 
          x = conv_silu<T>(a, vcol + d, t0 + t, off + t, p0 + t, start, slot, taps_end + (int64_t)(vcol + d) * a.taps);
        sv[t * ldv + d] = x;
      }
    }
  }
  if (warp == 0) {
    double lg = 0.0;
    float beta = 0.f;
    if (lane < n) {
      const float* gt = a.gates + (int64_t)(t0 + lane) * 2 * a.heads;
      beta = sigmoidf(gt[h]);
      lg = log_decay(gt[a.heads + h], a.dt_bias[h], a.a_log[h]);
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double x = __shfl_up_sync(0xffffffffu, lg, o);
      if (lane >= o) lg += x;
    }
    sL[lane] = lg;
    sB[lane] = beta;
    sE[lane] = expf((float)lg);
  }
  __syncthreads();
  // ---- unit vectors; the decayed copies go out right away
  const double lend = sL[kC - 1];
  for (int t = warp; t < kC; t += kThreads / 32) {
    float qq = 0.f, kk = 0.f;
    for (int d = lane; d < Dp; d += 32) {
      const float x = sq[t * ldk + d], y = sk[t * ldk + d];
      qq = fmaf(x, x, qq);
      kk = fmaf(y, y, kk);
    }
    const float iq = a.qscale / sqrtf(warp_sum(qq) + kUnitEps), ik = 1.0f / sqrtf(warp_sum(kk) + kUnitEps);
    const float gq = sE[t], gk = expf((float)(lend - sL[t]));
    for (int d = lane; d < Dp; d += 32) {
      const float x = sq[t * ldk + d] * iq, y = sk[t * ldk + d] * ik;
      sq[t * ldk + d] = x;
      sk[t * ldk + d] = y;
      out[L.q() + t * L.ldw + d] = x * gq;
      out[L.k() + t * L.ldk + d] = y * gk;
    }
  }
  if (tid == 0) out[L.g()] = expf((float)lend);
  __syncthreads();
  // ---- A (strictly below the diagonal) and P (with it): warp = one 16 x 8 tile of each
  {
    const int m0 = (warp >> 2) * 16, n0 = (warp & 3) * 8;
    Acc aa, pp;
    aa.zero();
    pp.zero();
    if (n0 <= m0 + 15) {
      for (int k0 = 0; k0 < Dp; k0 += 8) {
        const FragB b = frag_b([&](int k, int j) { return sk[(n0 + j) * ldk + k0 + k]; }, g, t4);
        aa.mac(frag_a([&](int r, int k) { return sk[(m0 + r) * ldk + k0 + k]; }, g, t4), b);
        pp.mac(frag_a([&](int r, int k) { return sq[(m0 + r) * ldk + k0 + k]; }, g, t4), b);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = m0 + g + 8 * (i >> 1), j = n0 + 2 * t4 + (i & 1);
      const float dec = j <= t ? expf((float)(sL[t] - sL[j])) : 0.f;
      sA[t * 36 + j] = j < t ? sB[t] * dec * aa.get(i) : 0.f;
      out[L.p() + t * L.ldp + j] = j <= t ? dec * pp.get(i) : 0.f;
    }
  }
  __syncthreads();
  // ---- inverse of I + A by halves: two warps solve the 16 x 16 blocks on the diagonal, a lane per column ...
  if (warp < 2) {
    const int b = warp * 16;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float r0 = t == lane ? 1.f : 0.f, r1 = 0.f, r2 = 0.f, r3 = 0.f;
#pragma unroll
      for (int i = 0; i < t; i += 4) {
        const float4 w = *reinterpret_cast<const float4*>(sA + (b + t) * 36 + b + i);
        r0 = fmaf(-w.x, x[i], r0);
        if (i + 1 < t) r1 = fmaf(-w.y, x[i + 1], r1);
        if (i + 2 < t) r2 = fmaf(-w.z, x[i + 2], r2);
        if (i + 3 < t) r3 = fmaf(-w.w, x[i + 3], r3);
      }
      x[t] = (r0 + r1) + (r2 + r3);
      if (lane < 16) sT[(b + t) * 36 + b + lane] = x[t];
    }
  }
  __syncthreads();
  // ... and the block below is -T22 (A21 T11), eight columns per warp (A11's place holds the product in between)
  if (warp < 2) {
    const int n0 = warp * 8;
    Acc acc;
    acc.zero();
#pragma unroll
    for (int k0 = 0; k0 < 16; k0 += 8)
      acc.mac(frag_a([&](int r, int k) { return sA[(16 + r) * 36 + k0 + k]; }, g, t4),
              frag_b([&](int k, int j) { return sT[(k0 + k) * 36 + n0 + j]; }, g, t4));
#pragma unroll
    for (int i = 0; i < 4; ++i) sA[(g + 8 * (i >> 1)) * 36 + n0 + 2 * t4 + (i & 1)] = acc.get(i);
    __syncwarp();
    acc.zero();
#pragma unroll
    for (int k0 = 0; k0 < 16; k0 += 8)
      acc.mac(frag_a([&](int r, int k) { return sT[(16 + r) * 36 + 16 + k0 + k]; }, g, t4),
              frag_b([&](int k, int j) { return sA[(k0 + k) * 36 + n0 + j]; }, g, t4));
#pragma unroll
    for (int i = 0; i < 4; ++i) sT[(16 + g + 8 * (i >> 1)) * 36 + n0 + 2 * t4 + (i & 1)] = -acc.get(i);
  }
  __syncthreads();
  // ---- W = T (beta e^L) K and Ub = T beta V: T's fragments stay in registers (its upper right block is zero), warps
  // take 8-wide column tiles
  FragA ft[6];                           // row tile 0: k 0, 8; row tile 1: k 0, 8, 16, 24
#pragma unroll
  for (int f = 0; f < 6; ++f) {
    const int m = f < 2 ? 0 : 16, k0 = (f < 2 ? f : f - 2) * 8;
    ft[f] = frag_a([&](int r, int k) { return sT[(m + r) * 36 + k0 + k] * sB[k0 + k]; }, g, t4);
  }
  const int nw = Dp / 8, ntile = nw + Vp / 8;
  for (int tile = warp; tile < ntile; tile += kThreads / 32) {
    const bool isw = tile < nw;
    const int n0 = (isw ? tile : tile - nw) * 8;
    const float* src = isw ? sk : sv;
    const int lds = isw ? ldk : ldv;
    Acc acc[2];
    acc[0].zero();
    acc[1].zero();
#pragma unroll
    for (int f = 0; f < 4; ++f) {
      const FragB b = frag_b([&](int k, int j) {
        const float y = src[(f * 8 + k) * lds + n0 + j];
        return isw ? y * sE[f * 8 + k] : y;
      }, g, t4);
      if (f < 2) acc[0].mac(ft[f], b);
      acc[1].mac(ft[2 + f], b);
    }
    float* dst = isw ? out + n0 : out + L.ub(n0 / kVS) + n0 % kVS;
    const int ldd = isw ? L.ldw : L.ldu;
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int i = 0; i < 4; i += 2)
        *reinterpret_cast<float2*>(dst + (m * 16 + g + 4 * i) * ldd + 2 * t4) =
            make_float2(acc[m].get(i), acc[m].get(i + 1));
  }
}

template <int MT>
__global__ void __launch_bounds__(kChunkThreads, 1) delta_chunks_kernel(ChunkArgs s, int stages) {
  constexpr int NW = kChunkThreads / 32, N1 = 16 / NW, N2 = 32 / NW;   // column tiles per warp: of [W; Q] S, of the state
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(8) uint64_t full[2];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kVS, nv = min(kVS, V - v0);
  const Scratch L(D, V);
  const int Dp = L.Dp, Dm = (D + 15) / 16 * 16, ldw = L.ldw, ldk = L.ldk, ldu = L.ldu;
  const int first = s.seq_chunk[seq], last = s.seq_chunk[seq + 1];
  const int ca = max(first, s.c0), cb = min(last, s.c1);
  if (ca >= cb) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* stage0 = sm;
  float* sS = stage0 + stages * L.stage();     // [Dm][40]
  float* sU = sS + Dm * ldu;                   // [32][40]
  const int row0 = a.seq_row[seq], len = a.seq_len[seq];
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0;

  struct View { const float *w, *q, *p, *ub, *k, *gc; };
  auto view = [&](int i) {
    const float* b = stage0 + (i % stages) * L.stage();
    return View{b, b + L.q(), b + L.p(), b + L.shared_part(), b + L.k(), b + L.g()};
  };
  auto fetch = [&](int c) {                    // one thread
    if (c >= cb) return;
    const float* src = s.scratch + ((int64_t)(c - s.c0) * a.heads + h) * L.floats();
    float* dst = stage0 + ((c - ca) % stages) * L.stage();
    uint64_t* bar = &full[(c - ca) % stages];
    tc5::mbar_expect_tx(bar, (uint32_t)(L.stage() * sizeof(float)));
    bulk_load(dst, src, (uint32_t)(L.shared_part() * sizeof(float)), bar);
    bulk_load(dst + L.shared_part(), src + L.ub(blockIdx.x), (uint32_t)(kC * ldu * sizeof(float)), bar);
  };

  if (tid == 0) {
    tc5::mbar_init(&full[0], 1);
    tc5::mbar_init(&full[1], 1);
    abort_word = 0;
    tc5::fence_barrier_init();
    for (int i = 0; i < stages; ++i) fetch(ca + i);
  }
  // ---- state: accumulator fragments of MT row tiles (eight apart), N2 column tiles each
  const int wm = warp / (4 / N2), wn = warp % (4 / N2) * N2;
  float S[MT][N2][4];
  const bool fresh = ca == first && p0 <= start;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < N2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (wm + 8 * m) * 16 + g + 8 * (i >> 1), c = (wn + n) * 8 + 2 * t4 + (i & 1);
        S[m][n][i] = !fresh && d < D && c < nv ? st[(int64_t)d * V + c] : 0.f;
        if (d < Dm) sS[d * ldu + c] = S[m][n][i];
      }

  const int mt = warp / (4 / N1), nt = warp % (4 / N1) * N1;           // row tile of [W; Q], first column tile
  bool ok = true;
  for (int c = ca; c < cb; ++c) {
    __syncthreads();                                   // the state is in place (and, first, the barriers)
    if (!tc5::mbar_wait(&full[(c - ca) % stages], ((c - ca) / stages) & 1, abort_flag)) {
      if (lane == 0) tc5::report(s.err, 40);
      ok = false;
      break;
    }
    const View v = view(c - ca);
    Acc acc[N1];
#pragma unroll
    for (int n = 0; n < N1; ++n) acc[n].zero();
    {
      const float* left = mt < 2 ? v.w + mt * 16 * ldw : v.q + (mt - 2) * 16 * ldw;
#pragma unroll 4
      for (int k0 = 0; k0 < Dp; k0 += 8) {
        const FragA fa = frag_a([&](int r, int k) { return left[r * ldw + k0 + k]; }, g, t4);
#pragma unroll
        for (int n = 0; n < N1; ++n)
          acc[n].mac(fa, frag_b([&](int k, int j) { return sS[(k0 + k) * ldu + (nt + n) * 8 + j]; }, g, t4));
      }
    }
    if (mt < 2) {
#pragma unroll
      for (int n = 0; n < N1; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int t = mt * 16 + g + 8 * (i >> 1), col = (nt + n) * 8 + 2 * t4 + (i & 1);
          sU[t * ldu + col] = v.ub[t * ldu + col] - acc[n].get(i);
        }
    }
    __syncthreads();                                   // U is complete, the old state is read
    if (mt >= 2) {
#pragma unroll
      for (int k0 = 0; k0 < kC; k0 += 8) {
        const FragA fa = frag_a([&](int r, int k) { return v.p[((mt - 2) * 16 + r) * L.ldp + k0 + k]; }, g, t4);
#pragma unroll
        for (int n = 0; n < N1; ++n)
          acc[n].mac(fa, frag_b([&](int k, int j) { return sU[(k0 + k) * ldu + (nt + n) * 8 + j]; }, g, t4));
      }
      const int off = (c - first) * kC;
#pragma unroll
      for (int n = 0; n < N1; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int t = off + (mt - 2) * 16 + g + 8 * (i >> 1), col = (nt + n) * 8 + 2 * t4 + (i & 1);
          if (t < len && col < nv) s.raw[((int64_t)(row0 + t) * a.heads + h) * V + v0 + col] = acc[n].get(i);
        }
    }
    const float gc = *v.gc;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int d0 = (wm + 8 * m) * 16;
      if (d0 < Dm) {
        Acc up[N2];
#pragma unroll
        for (int n = 0; n < N2; ++n) up[n].zero();
#pragma unroll
        for (int k0 = 0; k0 < kC; k0 += 8) {
          const FragA fa = frag_a([&](int r, int k) { return d0 + r < Dp ? v.k[(k0 + k) * ldk + d0 + r] : 0.f; }, g, t4);
#pragma unroll
          for (int n = 0; n < N2; ++n)
            up[n].mac(fa, frag_b([&](int k, int j) { return sU[(k0 + k) * ldu + (wn + n) * 8 + j]; }, g, t4));
        }
#pragma unroll
        for (int n = 0; n < N2; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            S[m][n][i] = fmaf(gc, S[m][n][i], up[n].get(i));
            sS[(d0 + g + 8 * (i >> 1)) * ldu + (wn + n) * 8 + 2 * t4 + (i & 1)] = S[m][n][i];
          }
      }
    }
    __syncthreads();                                   // the stage and U are free again
    if (tid == 0) fetch(c + stages);
  }
  if (!ok) {                                           // copies in flight still write to this CTA's memory
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
    for (int n = 0; n < N2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (wm + 8 * m) * 16 + g + 8 * (i >> 1), c = (wn + n) * 8 + 2 * t4 + (i & 1);
        if (d < D && c < nv) st[(int64_t)d * V + c] = S[m][n][i];
      }
}

bool sizes_ok(int heads, int kv_heads, int dim, int vdim, int taps) {
  return heads >= 1 && heads <= 65535 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 1 && dim <= 512 && vdim >= 1 &&
         vdim <= 65535 && taps >= 1;
}

Common common_args(const void* proj, int64_t ldp, const float* gates, const void* conv, const float* a_log,
                   const float* dt_bias, void* ring, float* state, const int* slot, const int* pos, const int* start,
                   const int* seq_row, const int* seq_len, int heads, int kv_heads, int dim, int vdim, int taps) {
  Common c = {proj, gates, conv, a_log, dt_bias, ring, state, slot, pos, start, seq_row, seq_len, ldp,
              heads, kv_heads, dim, vdim, taps, 2 * kv_heads * dim + heads * vdim, 1.0f / sqrtf((float)dim)};
  return c;
}

constexpr size_t kSmemMax = 226 * 1024;

template <typename T, int NR, int CV>
cudaError_t launch_step(const StepArgs& s, int seqs, bool fused, bool pdl, cudaStream_t st) {
  const int slices = (s.c.vdim + 32 * CV - 1) / (32 * CV);
  if (fused && slices > 8) return cudaErrorInvalidValue;
  const size_t smem = ((2 + s.c.taps) * (2 * (size_t)s.c.dim + 32 * CV) + 2 * 2 * 8 * 32 * CV) * sizeof(float);
  if (smem > kSmemMax) return cudaErrorInvalidValue;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(delta_step_kernel<T, NR, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
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
  return cudaLaunchKernelEx(&cfg, delta_step_kernel<T, NR, CV>, s);
}

// Columns per lane: as many as V divides into and the registers of NR rows leave room for, fewer while that spreads the
// large states of a few sequences over more SMs.
template <typename T, int NR>
cudaError_t pick_cols(const StepArgs& s, int seqs, bool fused, bool pdl, cudaStream_t st) {
  const int V = s.c.vdim;
  int cv = NR <= 16 && V % 4 == 0 && V > 64 ? 4 : NR <= 32 && V % 2 == 0 && V > 32 ? 2 : 1;
  while (cv > 1 && s.c.dim * 32 * cv > 4096 && (int64_t)s.c.heads * seqs * ((V + 16 * cv - 1) / (16 * cv)) <= 2 * 148) cv /= 2;
  if constexpr (NR <= 16)
    if (cv == 4) return launch_step<T, NR, 4>(s, seqs, fused, pdl, st);
  if constexpr (NR <= 32)
    if (cv == 2) return launch_step<T, NR, 2>(s, seqs, fused, pdl, st);
  return launch_step<T, NR, 1>(s, seqs, fused, pdl, st);
}

size_t prep_smem(const Scratch& L) {
  return (size_t)(2 * kC * (L.Dp + 4) + kC * (L.slices * kVS + 8) + 2 * kC * 36 + 4 * kC) * sizeof(float);
}
size_t chunk_smem(const Scratch& L, int D, int stages) {
  const int Dm = (D + 15) / 16 * 16;
  return ((size_t)(Dm + kC) * L.ldu + (size_t)stages * L.stage()) * sizeof(float);
}
}  // namespace

// Can the chunked form take these sizes?
IPEX_API int ipex_delta_chunks_ok(int dim, int vdim) {
  const Scratch L(dim, vdim);
  return dim >= 1 && dim <= 256 && vdim >= 1 && prep_smem(L) <= kSmemMax && chunk_smem(L, dim, 1) <= kSmemMax;
}
IPEX_API int64_t ipex_delta_scratch_floats(int dim, int vdim) { return Scratch(dim, vdim).floats(); }
// Can a decode step of these sizes norm its outputs on the way?
IPEX_API int ipex_delta_fused_ok(int vdim) { return vdim >= 1 && vdim <= 256; }

// Token by token.  seq_row / seq_len null: `seqs` sequences of one token each, whose convolution inputs are filed on
// the way; norm_w / out [tokens, ldo] then take the gated norm's result (vdim <= 256).  raw (when out is null): the
// plain outputs [tokens, heads, vdim].
IPEX_API int ipex_delta_step(const void* proj, int64_t ldp, int gate_off, const float* gates, const void* conv,
                             const float* a_log, const float* dt_bias, void* ring, float* state, const int* slot,
                             const int* pos, const int* start, const int* seq_row, const int* seq_len, int seqs,
                             const void* norm_w, float eps, void* out, int64_t ldo, float* raw, int heads, int kv_heads,
                             int dim, int vdim, int taps, int dtype, int pdl, void* stream) {
  if (!sizes_ok(heads, kv_heads, dim, vdim, taps) || seqs < 1 || seqs > 65535 || (seq_row == nullptr) != (seq_len == nullptr))
    return (int)cudaErrorInvalidValue;
  const bool fused = raw == nullptr;
  if (fused && (seq_row != nullptr || out == nullptr || norm_w == nullptr || !ipex_delta_fused_ok(vdim)))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    StepArgs s = {common_args(proj, ldp, gates, conv, a_log, dt_bias, ring, state, slot, pos, start, seq_row, seq_len,
                              heads, kv_heads, dim, vdim, taps),
                  norm_w, out, raw, ldo, eps, gate_off, seq_row == nullptr, pdl && fused && vdim % 4 == 0};
    cudaStream_t st = (cudaStream_t)stream;
    if (dim <= 32) return pick_cols<T, 4>(s, seqs, fused, pdl != 0, st);
    if (dim <= 64) return pick_cols<T, 8>(s, seqs, fused, pdl != 0, st);
    if (dim <= 128) return pick_cols<T, 16>(s, seqs, fused, pdl != 0, st);
    if (dim <= 256) return pick_cols<T, 32>(s, seqs, fused, pdl != 0, st);
    return pick_cols<T, 64>(s, seqs, fused, pdl != 0, st);
  });
}

// Chunks [c0, c1) of a packed batch in the chunked form (16-bit models).  chunk_seq [chunks], seq_chunk [seqs + 1]: device tables of the
// sequences' chunks of 32 tokens, in order; scratch: (c1 - c0) * heads * ipex_delta_scratch_floats; raw as above.
IPEX_API int ipex_delta_chunks(const void* proj, int64_t ldp, const float* gates, const void* conv, const float* a_log,
                               const float* dt_bias, void* ring, float* state, const int* slot, const int* pos,
                               const int* start, const int* seq_row, const int* seq_len, int seqs, const int* chunk_seq,
                               const int* seq_chunk, int c0, int c1, float* scratch, float* raw, int heads, int kv_heads,
                               int dim, int vdim, int taps, int dtype, int* err, void* stream) {
  if (!sizes_ok(heads, kv_heads, dim, vdim, taps) || !ipex_delta_chunks_ok(dim, vdim) || seqs < 1 || seqs > 65535 ||
      c0 < 0 || c1 <= c0 || seq_row == nullptr || seq_len == nullptr || (((uintptr_t)scratch) & 15) || dtype == DT_F32)
    return (int)cudaErrorInvalidValue;
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ChunkArgs s = {common_args(proj, ldp, gates, conv, a_log, dt_bias, ring, state, slot, pos, start, seq_row, seq_len,
                               heads, kv_heads, dim, vdim, taps),
                   chunk_seq, seq_chunk, scratch, raw, err, c0, c1, 0};
    // 16-byte reads, and room for the convolution weights where A and its inverse go later
    s.vec = dim % 8 == 0 && vdim % 8 == 0 && ldp % 8 == 0 && (((uintptr_t)proj | (uintptr_t)ring) & 15) == 0 &&
            (2 * dim + vdim) * taps <= 2 * kC * 36;
    cudaStream_t st = (cudaStream_t)stream;
    const Scratch L(dim, vdim);
    const size_t ps = prep_smem(L);
    auto prep = taps == 4 ? delta_prep_kernel<T, 4> : delta_prep_kernel<T, 0>;
    cudaError_t e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ps);
    if (e != cudaSuccess) return e;
    prep<<<dim3(c1 - c0, heads), kThreads, ps, st>>>(s);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const int stages = chunk_smem(L, dim, 2) <= kSmemMax ? 2 : 1;
    const size_t cs = chunk_smem(L, dim, stages);
    auto kern = dim <= 128 ? delta_chunks_kernel<1> : delta_chunks_kernel<2>;
    e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cs);
    if (e != cudaSuccess) return e;
    kern<<<dim3(L.slices, heads, seqs), kChunkThreads, cs, st>>>(s, stages);
    return cudaGetLastError();
  };
  return (int)(dtype == DT_F16 ? run((__half*)nullptr) : run((__nv_bfloat16*)nullptr));
}
