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
//   delta_tail    the last inputs of the convolutions into the slot's ring
//   gated_norm    o / rms(o) * w * silu(gate) behind delta_chunks
//
// The products of the chunked form run on the tensor cores with every fp32 operand split into two tf32 parts (three
// products, about 22 bits), accumulated in fp32; the state itself is only ever added to in fp32.  The state's columns
// are independent, so a head is spread over slices of 32 columns.
//
// Convolution inputs are kept in a ring of `taps` rows per slot (row = position mod taps): a decode step writes a row
// that no other block of the step reads.  What lies before a sequence's first token counts as zero, and so does the
// state there, so a slot needs no clearing when it changes hands.
#include <cooperative_groups.h>

#include "common/utils.cuh"

namespace {

namespace cg = cooperative_groups;

constexpr int kThreads = 256;
constexpr int kC = 32;                // tokens per chunk
constexpr int kVS = 32;               // state columns per CTA

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

// Channel c of the convolution at packed token t (position p), after silu.
template <typename T>
__device__ __forceinline__ float conv_silu(const Common& a, int c, int t, int row0, int p, int start, int slot) {
  const T* proj = reinterpret_cast<const T*>(a.proj);
  const T* w = reinterpret_cast<const T*>(a.conv) + (int64_t)c * a.taps;
  const T* ring = reinterpret_cast<const T*>(a.ring) + (int64_t)slot * a.taps * a.channels + c;
  float s = 0.f;
  for (int i = 0; i < a.taps; ++i) {
    const int back = a.taps - 1 - i;
    if (p - back < start) continue;
    const float x = t - back >= row0 ? DT<T>::to_f(proj[(int64_t)(t - back) * a.ldp + c])
                                     : DT<T>::to_f(ring[(int64_t)((p - back) % a.taps) * a.channels]);
    s = fmaf(x, DT<T>::to_f(w[i]), s);
  }
  return silu(s);
}

// log of the decay and write strength of one token and head
__device__ __forceinline__ float log_decay(float a, float dt_bias, float a_log) {
  const float z = a + dt_bias;
  const float sp = z > 20.f ? z : log1pf(expf(z));
  return -expf(a_log) * sp;
}
__device__ __forceinline__ float sigmoidf(float x) { return 1.0f / (1.0f + expf(-x)); }

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
};

// A warp owns the state rows warp, warp + 8, ...; a lane one of 32 columns.
template <typename T, int NR>
__global__ void __launch_bounds__(kThreads) delta_step_kernel(StepArgs s) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, sq_id = blockIdx.z, slice = blockIdx.x;
  const int hk = h / (a.heads / a.kv_heads), v0 = slice * kVS, nv = min(kVS, V - v0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* buf = sm;                      // [2][2 D + 32]: q, k, v of a token
  float* red = buf + 2 * (2 * D + kVS); // [2][2][8][32]
  __shared__ float s_ss;
  const int row0 = a.seq_row != nullptr ? a.seq_row[sq_id] : sq_id, len = a.seq_len != nullptr ? a.seq_len[sq_id] : 1;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0 + lane;
  float S[NR];
  const bool fresh = p0 <= start, col = lane < nv;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = warp + 8 * i;
    S[i] = !fresh && col && d < D ? st[(int64_t)d * V] : 0.f;
  }
  const int qc = hk * D, kc = a.kv_heads * D + hk * D, vc = 2 * a.kv_heads * D + h * V + v0;
  const float alog = a.a_log[h], dtb = a.dt_bias[h];
  for (int j = 0; j < len; ++j) {
    const int t = row0 + j, p = p0 + j;
    float* q = buf + (j & 1) * (2 * D + kVS);
    float* k = q + D;
    float* v = k + D;
    float* rd = red + (j & 1) * (2 * 8 * 32);
    for (int i = tid; i < 2 * D + nv; i += kThreads) {
      const int c = i < D ? qc + i : i < 2 * D ? kc + i - D : vc + i - 2 * D;
      q[i] = conv_silu<T>(a, c, t, row0, p, start, slot);
    }
    const float beta = sigmoidf(a.gates[(int64_t)t * 2 * a.heads + h]);
    const float g = expf(log_decay(a.gates[(int64_t)t * 2 * a.heads + a.heads + h], dtb, alog));
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int d = lane; d < D; d += 32) {
      qq = fmaf(q[d], q[d], qq);
      kk = fmaf(k[d], k[d], kk);
      qk = fmaf(q[d], k[d], qk);
    }
    const float iq = a.qscale / sqrtf(warp_sum(qq) + kUnitEps), ik = 1.0f / sqrtf(warp_sum(kk) + kUnitEps);
    qk = warp_sum(qk) * iq * ik;
    float sk = 0.f, sq = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        sk = fmaf(S[i], k[d], sk);
        sq = fmaf(S[i], q[d], sq);
      }
    }
    rd[warp * 32 + lane] = sk;
    rd[(8 + warp) * 32 + lane] = sq;
    __syncthreads();
    sk = sq = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      sk += rd[w * 32 + lane];
      sq += rd[(8 + w) * 32 + lane];
    }
    const float u = col ? beta * (v[lane] - g * ik * sk) : 0.f;
    const float o = g * iq * sq + qk * u;            // S^T q after the write
    const float ku = ik * u;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) S[i] = fmaf(k[d], ku, g * S[i]);
    }
    if (s.raw != nullptr) {
      if (warp == 0 && col) s.raw[((int64_t)t * a.heads + h) * V + v0 + lane] = o;
    } else {
      // one token: norm over all columns of the head, which the CTAs of the cluster hold slice by slice
      const float ss = warp_sum(o * o);
      if (tid == 0) s_ss = ss;
      float total = ss;
      if (gridDim.x > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        cluster.sync();
        total = 0.f;
        for (int r = 0; r < (int)gridDim.x; ++r) total += *cluster.map_shared_rank(&s_ss, r);
        cluster.sync();
      }
      if (warp == 0 && col) {
        const float inv = 1.0f / sqrtf(total / (float)V + s.eps);
        const int c = h * V + v0 + lane;
        const float gate = DT<T>::to_f(reinterpret_cast<const T*>(a.proj)[(int64_t)t * a.ldp + s.gate_off + c]);
        const float w = DT<T>::to_f(reinterpret_cast<const T*>(s.norm_w)[v0 + lane]);
        reinterpret_cast<T*>(s.out)[(int64_t)t * s.ldo + c] = DT<T>::from_f(o * inv * w * silu(gate));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = warp + 8 * i;
    if (col && d < D) st[(int64_t)d * V] = S[i];
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
    if (tid < nv) ring[vc + tid] = proj[vc + tid];
  }
}

// ---------------------------------------------------------------------------------------------- tf32 pairs
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xFFFFE000u;
  lo = __float_as_uint(x - __uint_as_float(hi)) & 0xFFFFE000u;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
struct FragA { uint32_t hi[4], lo[4]; };
struct FragB { uint32_t hi[2], lo[2]; };
// lane (g, t): A rows g, g + 8 and columns t, t + 4; B row (k) t, t + 4 of column g; C rows g, g + 8, columns 2t, 2t + 1
template <typename F>
__device__ __forceinline__ FragA frag_a(F&& at, int g, int t) {
  FragA f;
  split_tf32(at(g, t), f.hi[0], f.lo[0]);
  split_tf32(at(g + 8, t), f.hi[1], f.lo[1]);
  split_tf32(at(g, t + 4), f.hi[2], f.lo[2]);
  split_tf32(at(g + 8, t + 4), f.hi[3], f.lo[3]);
  return f;
}
template <typename F>
__device__ __forceinline__ FragB frag_b(F&& at, int g, int t) {
  FragB f;
  split_tf32(at(t, g), f.hi[0], f.lo[0]);
  split_tf32(at(t + 4, g), f.hi[1], f.lo[1]);
  return f;
}
// independent accumulators for the main and the two correction products: three short chains instead of a long one
struct Acc {
  float m[4], x[4], y[4];
  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int i = 0; i < 4; ++i) m[i] = x[i] = y[i] = 0.f;
  }
  __device__ __forceinline__ void mac(const FragA& a, const FragB& b) {
    mma_tf32(m, a.hi, b.hi);
    mma_tf32(x, a.hi, b.lo);
    mma_tf32(y, a.lo, b.hi);
  }
  __device__ __forceinline__ float get(int i) const { return m[i] + (x[i] + y[i]); }
};

// Scratch of one (chunk, head): W, Q and K parts [32][Dp] each, P [32][32], Ub [32][Vp], decay of the whole chunk
struct Scratch {
  int Dp, Vp;
  __host__ __device__ Scratch(int D, int V) : Dp((D + 7) / 8 * 8), Vp((V + kVS - 1) / kVS * kVS) {}
  __host__ __device__ int64_t floats() const { return (int64_t)kC * (3 * Dp + kC + Vp) + 4; }
  __host__ __device__ int64_t w() const { return 0; }
  __host__ __device__ int64_t q() const { return (int64_t)kC * Dp; }
  __host__ __device__ int64_t k() const { return (int64_t)kC * 2 * Dp; }
  __host__ __device__ int64_t p() const { return (int64_t)kC * 3 * Dp; }
  __host__ __device__ int64_t ub() const { return p() + kC * kC; }
  __host__ __device__ int64_t g() const { return ub() + (int64_t)kC * Vp; }
};

struct ChunkArgs {
  Common c;
  const int* chunk_seq;     // [all chunks] sequence of a chunk
  const int* seq_chunk;     // [sequences + 1] first chunk of a sequence
  float* scratch;           // of the chunks [c0, c1), [chunk - c0][head]
  float* raw;               // o [tokens, heads, vdim]
  int c0, c1;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) delta_prep_kernel(ChunkArgs s) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, chunk = s.c0 + blockIdx.x;
  const Scratch L(D, V);
  const int Dp = L.Dp, Vp = L.Vp, ldk = Dp + 4, ldv = Vp + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* sq = sm;                        // [32][Dp + 4]
  float* sk = sq + kC * ldk;             // [32][Dp + 4]
  float* sv = sk + kC * ldk;             // [32][Vp + 8]
  float* sA = sv + kC * ldv;             // [32][36]
  float* sT = sA + kC * 36;              // [32][36]
  // [32] running sum of log g, in 64-bit: its differences must keep 32-bit accuracy when single tokens decay to nothing
  double* sL = reinterpret_cast<double*>(sT + kC * 36);
  float* sB = reinterpret_cast<float*>(sL + kC);      // [32] beta
  const int seq = s.chunk_seq[chunk], hk = h / (a.heads / a.kv_heads);
  const int row0 = a.seq_row[seq], off = (chunk - s.seq_chunk[seq]) * kC, n = min(kC, a.seq_len[seq] - off);
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0] + off, t0 = row0 + off;
  float* out = s.scratch + ((int64_t)(chunk - s.c0) * a.heads + h) * L.floats();
  const int qc = hk * D, kcol = a.kv_heads * D + hk * D, vcol = 2 * a.kv_heads * D + h * V;

  // ---- convolutions (zeros behind the sequence's end and past the sizes)
  const int per = 2 * Dp + Vp;
  for (int i = tid; i < kC * per; i += kThreads) {
    const int t = i / per, c = i % per;
    float x = 0.f;
    if (c < 2 * Dp) {
      const int d = c < Dp ? c : c - Dp;
      if (t < n && d < D) x = conv_silu<T>(a, (c < Dp ? qc : kcol) + d, t0 + t, row0, p0 + t, start, slot);
      (c < Dp ? sq : sk)[t * ldk + d] = x;
    } else {
      const int d = c - 2 * Dp;
      if (t < n && d < V) x = conv_silu<T>(a, vcol + d, t0 + t, row0, p0 + t, start, slot);
      sv[t * ldv + d] = x;
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
    const float gq = expf((float)sL[t]), gk = expf((float)(lend - sL[t]));
    for (int d = lane; d < Dp; d += 32) {
      const float x = sq[t * ldk + d] * iq, y = sk[t * ldk + d] * ik;
      sq[t * ldk + d] = x;
      sk[t * ldk + d] = y;
      out[L.q() + t * Dp + d] = x * gq;
      out[L.k() + t * Dp + d] = y * gk;
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
      out[L.p() + t * kC + j] = j <= t ? dec * pp.get(i) : 0.f;
    }
  }
  __syncthreads();
  // ---- inverse of I + A: lane j solves for column j
  if (warp == 0) {
    float x[kC];
#pragma unroll
    for (int t = 0; t < kC; ++t) {
      float r0 = t == lane ? 1.f : 0.f, r1 = 0.f, r2 = 0.f, r3 = 0.f;
#pragma unroll
      for (int i = 0; i < t; i += 4) {
        const float4 w = *reinterpret_cast<const float4*>(sA + t * 36 + i);
        r0 = fmaf(-w.x, x[i], r0);
        if (i + 1 < t) r1 = fmaf(-w.y, x[i + 1], r1);
        if (i + 2 < t) r2 = fmaf(-w.z, x[i + 2], r2);
        if (i + 3 < t) r3 = fmaf(-w.w, x[i + 3], r3);
      }
      x[t] = (r0 + r1) + (r2 + r3);
      sT[t * 36 + lane] = x[t] * sB[lane];      // column j times beta_j: the right-hand sides carry it
    }
  }
  __syncthreads();
  // ---- W = T (beta e^L) K and Ub = T beta V: warps take 8-wide column tiles, both row tiles
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
    for (int k0 = 0; k0 < kC; k0 += 8) {
      const FragB b = frag_b([&](int k, int j) {
        const float y = src[(k0 + k) * lds + n0 + j];
        return isw ? y * expf((float)sL[k0 + k]) : y;
      }, g, t4);
#pragma unroll
      for (int m = 0; m < 2; ++m)
        acc[m].mac(frag_a([&](int r, int k) { return sT[(m * 16 + r) * 36 + k0 + k]; }, g, t4), b);
    }
    float* dst = isw ? out + L.w() : out + L.ub();
    const int ldd = isw ? Dp : Vp;
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int i = 0; i < 4; i += 2)
        *reinterpret_cast<float2*>(dst + (m * 16 + g + 4 * i) * ldd + n0 + 2 * t4) =
            make_float2(acc[m].get(i), acc[m].get(i + 1));
  }
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

template <int MT>
__global__ void __launch_bounds__(kThreads, 1) delta_chunks_kernel(ChunkArgs s, int stages) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kVS, nv = min(kVS, V - v0);
  const Scratch L(D, V);
  const int Dp = L.Dp, Dm = (D + 15) / 16 * 16, ldw = Dp + 4, ldk = Dp + 8, ldu = 40;
  const int first = s.seq_chunk[seq], last = s.seq_chunk[seq + 1];
  const int ca = max(first, s.c0), cb = min(last, s.c1);
  if (ca >= cb) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int stage_floats = kC * (2 * ldw + 36 + 40) + kC * ldk + 8;
  float* sS = sm;                              // [Dm][40]
  float* sU = sS + Dm * ldu;                   // [32][40]
  float* stage0 = sU + kC * ldu;
  const int row0 = a.seq_row[seq], len = a.seq_len[seq];
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0;

  struct View { float *w, *q, *p, *ub, *k, *gc; };
  auto view = [&](int i) {
    float* b = stage0 + (i % stages) * stage_floats;
    View v;
    v.w = b;
    v.q = v.w + kC * ldw;
    v.p = v.q + kC * ldw;
    v.ub = v.p + kC * 36;
    v.k = v.ub + kC * 40;
    v.gc = v.k + kC * ldk;
    return v;
  };
  auto fetch = [&](int c) {
    if (c < cb) {
      const float* src = s.scratch + ((int64_t)(c - s.c0) * a.heads + h) * L.floats();
      const View v = view(c - ca);
      const int nd = Dp / 4;
      for (int i = tid; i < kC * nd; i += kThreads) {
        const int t = i / nd, d = (i % nd) * 4;
        cp_async16(v.w + t * ldw + d, src + L.w() + t * Dp + d);
        cp_async16(v.q + t * ldw + d, src + L.q() + t * Dp + d);
        cp_async16(v.k + t * ldk + d, src + L.k() + t * Dp + d);
      }
      for (int i = tid; i < kC * 8; i += kThreads) {
        const int t = i / 8, d = (i % 8) * 4;
        cp_async16(v.p + t * 36 + d, src + L.p() + t * kC + d);
        cp_async16(v.ub + t * 40 + d, src + L.ub() + t * L.Vp + v0 + d);
      }
      if (tid == 0) cp_async16(v.gc, src + L.g());
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  fetch(ca);
  // ---- state: accumulator fragments of the row tiles warp, warp + 8, ... (MT of them)
  float S[MT][4][4];
  const bool fresh = ca == first && p0 <= start;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (warp + 8 * m) * 16 + g + 8 * (i >> 1), c = n * 8 + 2 * t4 + (i & 1);
        S[m][n][i] = !fresh && d < D && c < nv ? st[(int64_t)d * V + c] : 0.f;
        if (d < Dm) sS[d * ldu + c] = S[m][n][i];
      }

  const int mt = warp >> 1, nt0 = (warp & 1) * 2;      // row tile of [W; Q], first of two column tiles
  for (int c = ca; c < cb; ++c) {
    if (stages > 1) {
      fetch(c + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();                                   // this chunk's parts and the state are in place
    const View v = view(c - ca);
    Acc acc[2];
    acc[0].zero();
    acc[1].zero();
    {
      const float* left = mt < 2 ? v.w + mt * 16 * ldw : v.q + (mt - 2) * 16 * ldw;
#pragma unroll 4
      for (int k0 = 0; k0 < Dp; k0 += 8) {
        const FragA fa = frag_a([&](int r, int k) { return left[r * ldw + k0 + k]; }, g, t4);
#pragma unroll
        for (int n = 0; n < 2; ++n)
          acc[n].mac(fa, frag_b([&](int k, int j) { return sS[(k0 + k) * ldu + (nt0 + n) * 8 + j]; }, g, t4));
      }
    }
    if (mt < 2) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int t = mt * 16 + g + 8 * (i >> 1), col = (nt0 + n) * 8 + 2 * t4 + (i & 1);
          sU[t * ldu + col] = v.ub[t * 40 + col] - acc[n].get(i);
        }
    }
    __syncthreads();                                   // U is complete, the old state is read
    if (mt >= 2) {
#pragma unroll
      for (int k0 = 0; k0 < kC; k0 += 8) {
        const FragA fa = frag_a([&](int r, int k) { return v.p[((mt - 2) * 16 + r) * 36 + k0 + k]; }, g, t4);
#pragma unroll
        for (int n = 0; n < 2; ++n)
          acc[n].mac(fa, frag_b([&](int k, int j) { return sU[(k0 + k) * ldu + (nt0 + n) * 8 + j]; }, g, t4));
      }
      const int off = (c - first) * kC;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int t = off + (mt - 2) * 16 + g + 8 * (i >> 1), col = (nt0 + n) * 8 + 2 * t4 + (i & 1);
          if (t < len && col < nv) s.raw[((int64_t)(row0 + t) * a.heads + h) * V + v0 + col] = acc[n].get(i);
        }
    }
    const float gc = *v.gc;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int d0 = (warp + 8 * m) * 16;
      if (d0 < Dm) {
        Acc up[4];
#pragma unroll
        for (int n = 0; n < 4; ++n) up[n].zero();
#pragma unroll
        for (int k0 = 0; k0 < kC; k0 += 8) {
          const FragA fa = frag_a([&](int r, int k) { return d0 + r < Dp ? v.k[(k0 + k) * ldk + d0 + r] : 0.f; }, g, t4);
#pragma unroll
          for (int n = 0; n < 4; ++n)
            up[n].mac(fa, frag_b([&](int k, int j) { return sU[(k0 + k) * ldu + n * 8 + j]; }, g, t4));
        }
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            S[m][n][i] = fmaf(gc, S[m][n][i], up[n].get(i));
            sS[(d0 + g + 8 * (i >> 1)) * ldu + n * 8 + 2 * t4 + (i & 1)] = S[m][n][i];
          }
      }
    }
    __syncthreads();                                   // the stage and U are free again
    if (stages == 1) fetch(c + 1);
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (warp + 8 * m) * 16 + g + 8 * (i >> 1), c = n * 8 + 2 * t4 + (i & 1);
        if (d < D && c < nv) st[(int64_t)d * V + c] = S[m][n][i];
      }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

template <typename T>
__global__ void __launch_bounds__(kThreads) delta_tail_kernel(Common a) {
  const int seq = blockIdx.y, len = a.seq_len[seq], row0 = a.seq_row[seq], n = min(len, a.taps);
  const int c = blockIdx.x * kThreads + threadIdx.x, slot = a.slot[row0], p0 = a.pos[row0];
  if (c >= a.channels) return;
  T* ring = reinterpret_cast<T*>(a.ring) + (int64_t)slot * a.taps * a.channels + c;
  const T* proj = reinterpret_cast<const T*>(a.proj) + c;
  for (int j = len - n; j < len; ++j)
    ring[(int64_t)((p0 + j) % a.taps) * a.channels] = proj[(int64_t)(row0 + j) * a.ldp];
}

// A warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(kThreads) gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate,
                                                              int64_t ldg, const T* __restrict__ w, T* __restrict__ out,
                                                              int64_t ldo, int64_t rows, int heads, int V, float eps) {
  const int64_t r = (int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= rows) return;
  const int64_t t = r / heads;
  const int h = (int)(r % heads);
  const float* src = o + r * V;
  float ss = 0.f;
  for (int i = lane; i < V; i += 32) ss = fmaf(src[i], src[i], ss);
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps);
  for (int i = lane; i < V; i += 32)
    out[t * ldo + h * V + i] =
        DT<T>::from_f(src[i] * inv * DT<T>::to_f(w[i]) * silu(DT<T>::to_f(gate[t * ldg + h * V + i])));
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

template <typename T, int NR>
cudaError_t launch_step(const StepArgs& s, int seqs, bool fused, bool pdl, cudaStream_t st) {
  const int slices = (s.c.vdim + kVS - 1) / kVS;
  const size_t smem = (2 * (2 * (size_t)s.c.dim + kVS) + 2 * 2 * 8 * 32) * sizeof(float);
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
  return cudaLaunchKernelEx(&cfg, delta_step_kernel<T, NR>, s);
}

size_t prep_smem(const Scratch& L) {
  return (size_t)(2 * kC * (L.Dp + 4) + kC * (L.Vp + 8) + 2 * kC * 36 + 3 * kC) * sizeof(float);
}
size_t chunk_smem(const Scratch& L, int D, int stages) {
  const int Dm = (D + 15) / 16 * 16;
  return ((size_t)(Dm + kC) * 40 +
          (size_t)stages * (kC * (2 * (L.Dp + 4) + 36 + 40) + kC * (L.Dp + 8) + 8)) * sizeof(float);
}
constexpr size_t kSmemMax = 226 * 1024;

}  // namespace

// Can the chunked form take these sizes?
IPEX_API int ipex_delta_chunks_ok(int dim, int vdim) {
  const Scratch L(dim, vdim);
  return dim >= 1 && dim <= 256 && vdim >= 1 && prep_smem(L) <= kSmemMax && chunk_smem(L, dim, 1) <= kSmemMax;
}
IPEX_API int64_t ipex_delta_scratch_floats(int dim, int vdim) { return Scratch(dim, vdim).floats(); }
// Column slices of a head: the fused norm of a decode step takes up to eight.
IPEX_API int ipex_delta_slices(int vdim) { return (vdim + kVS - 1) / kVS; }

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
  if (fused && (seq_row != nullptr || out == nullptr || norm_w == nullptr || ipex_delta_slices(vdim) > 8))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    StepArgs s = {common_args(proj, ldp, gates, conv, a_log, dt_bias, ring, state, slot, pos, start, seq_row, seq_len,
                              heads, kv_heads, dim, vdim, taps),
                  norm_w, out, raw, ldo, eps, gate_off, seq_row == nullptr};
    cudaStream_t st = (cudaStream_t)stream;
    if (dim <= 32) return launch_step<T, 4>(s, seqs, fused, pdl != 0, st);
    if (dim <= 64) return launch_step<T, 8>(s, seqs, fused, pdl != 0, st);
    if (dim <= 128) return launch_step<T, 16>(s, seqs, fused, pdl != 0, st);
    if (dim <= 256) return launch_step<T, 32>(s, seqs, fused, pdl != 0, st);
    return launch_step<T, 64>(s, seqs, fused, pdl != 0, st);
  });
}

// Chunks [c0, c1) of a packed batch in the chunked form (16-bit models).  chunk_seq [chunks], seq_chunk [seqs + 1]: device tables of the
// sequences' chunks of 32 tokens, in order; scratch: (c1 - c0) * heads * ipex_delta_scratch_floats; raw as above.
IPEX_API int ipex_delta_chunks(const void* proj, int64_t ldp, const float* gates, const void* conv, const float* a_log,
                               const float* dt_bias, void* ring, float* state, const int* slot, const int* pos,
                               const int* start, const int* seq_row, const int* seq_len, int seqs, const int* chunk_seq,
                               const int* seq_chunk, int c0, int c1, float* scratch, float* raw, int heads, int kv_heads,
                               int dim, int vdim, int taps, int dtype, void* stream) {
  if (!sizes_ok(heads, kv_heads, dim, vdim, taps) || !ipex_delta_chunks_ok(dim, vdim) || seqs < 1 || seqs > 65535 ||
      c0 < 0 || c1 <= c0 || seq_row == nullptr || seq_len == nullptr || (((uintptr_t)scratch) & 15) || dtype == DT_F32)
    return (int)cudaErrorInvalidValue;
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ChunkArgs s = {common_args(proj, ldp, gates, conv, a_log, dt_bias, ring, state, slot, pos, start, seq_row, seq_len,
                               heads, kv_heads, dim, vdim, taps),
                   chunk_seq, seq_chunk, scratch, raw, c0, c1};
    cudaStream_t st = (cudaStream_t)stream;
    const Scratch L(dim, vdim);
    const size_t ps = prep_smem(L);
    cudaError_t e = cudaFuncSetAttribute(delta_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ps);
    if (e != cudaSuccess) return e;
    delta_prep_kernel<T><<<dim3(c1 - c0, heads), kThreads, ps, st>>>(s);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const int stages = chunk_smem(L, dim, 2) <= kSmemMax ? 2 : 1;
    const size_t cs = chunk_smem(L, dim, stages);
    auto kern = dim <= 128 ? delta_chunks_kernel<1> : delta_chunks_kernel<2>;
    e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cs);
    if (e != cudaSuccess) return e;
    kern<<<dim3(ipex_delta_slices(vdim), heads, seqs), kThreads, cs, st>>>(s, stages);
    return cudaGetLastError();
  };
  return (int)(dtype == DT_F16 ? run((__half*)nullptr) : run((__nv_bfloat16*)nullptr));
}

// The last convolution inputs of every sequence into its slot's ring (after everything that reads the ring).
IPEX_API int ipex_delta_tail(const void* proj, int64_t ldp, void* ring, const int* slot, const int* pos,
                             const int* seq_row, const int* seq_len, int seqs, int channels, int taps, int dtype,
                             void* stream) {
  if (seqs < 1 || seqs > 65535 || channels < 1 || taps < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    Common c = {};
    c.proj = proj; c.ldp = ldp; c.ring = ring; c.slot = slot; c.pos = pos; c.seq_row = seq_row; c.seq_len = seq_len;
    c.channels = channels; c.taps = taps;
    delta_tail_kernel<T><<<dim3((channels + kThreads - 1) / kThreads, seqs), kThreads, 0, (cudaStream_t)stream>>>(c);
    return cudaGetLastError();
  });
}

// out[t, h, :] = o / sqrt(mean(o^2) + eps) * w * silu(gate), o [tokens, heads, vdim] fp32
IPEX_API int ipex_gated_norm(const float* o, const void* gate, int64_t ldg, const void* w, void* out, int64_t ldo,
                             int tokens, int heads, int vdim, float eps, int dtype, void* stream) {
  if (tokens < 1 || heads < 1 || vdim < 1) return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int64_t rows = (int64_t)tokens * heads;
    gated_norm_kernel<T><<<(unsigned)((rows + 7) / 8), kThreads, 0, (cudaStream_t)stream>>>(
        o, (const T*)gate, ldg, (const T*)w, (T*)out, ldo, rows, heads, vdim, eps);
    return cudaGetLastError();
  });
}
