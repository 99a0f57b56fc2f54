// State-space duality (selective state spaces with a scalar decay per head), sm_100a.
//
// Per head a matrix state S [state, vdim] is carried from token to token:
//     S <- exp(-e^A dt) S + dt B x^T;   y = S^T C + D x        dt = softplus(. + bias)
// x (per head), B and C (shared by groups of heads) come from projections through a causal convolution over a few tokens
// (per channel, with a bias) and silu; dt from a projection.  dt, the decay, B, C, the state and the products that touch it
// are fp32; x has the activation dtype.
//
//   ssd_step    token by token, state in registers: decoding (one token of every sequence), short portions, 32-bit models
//   ssd_groups  prompts, parallel over chunks of 32 tokens and groups: B, C, and their products C . B
//   ssd_heads   prompts, parallel over chunks and heads: x, and with L the running sum of the decays' logarithms
//               P[t,i] = e^(L_t - L_i) dt_i (C_t . B_i) for i <= t, read factors e^L_t, write factors e^(L_end - L_i) dt_i
//   ssd_chunks  prompts, sequential over a sequence's chunks: Y = e^L (C S) + P X + D X, S <- e^L_end S + (f B)^T X
//
// Products of the chunked form run on the tensor cores with fp32 operands split into tf32 pairs (x is exact in one part).
// The state lives transposed in accumulator fragments, which serve as the left operand of the next chunk's read-out.
//
// What lies before a sequence's first token counts as zero, so a slot needs no clearing when it changes hands.
#include "common/short_conv.cuh"
#include "common/state_cols.cuh"
#include "common/tf32_pairs.cuh"
#include "common/utils.cuh"
#include "tcgen05_common.cuh"

namespace {

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
  const void* proj;       // T [tokens, ldp]: x heads, B groups, C groups (the convolved channels)
  const float* dt;        // [tokens, ldt], the first `heads` columns
  const void* conv;       // T [channels, taps]
  const float* conv_b;    // [channels]
  const float* dt_bias;   // [heads]
  const float* a_log;     // [heads]
  const float* skip;      // [heads]: D
  void* ring;             // T [slots, taps, channels]
  float* state;           // [slots, heads, dim, vdim]
  const int* slot;        // [tokens]
  const int* pos;         // [tokens]
  const int* start;       // [slots]
  const int* seq_row;     // [sequences] first packed token, or null: sequence = token
  const int* seq_len;
  int64_t ldp, ldt;
  int heads, groups, dim, vdim, taps, channels;
};

template <typename T>
__device__ __forceinline__ float rounded(float v) { return DT<T>::to_f(DT<T>::from_f(v)); }

// ---------------------------------------------------------------------------------------------- token by token
struct StepArgs {
  Common c;
  float* raw;             // y [tokens, heads, vdim]
  int ring_write;         // one token per sequence: file its convolution inputs
  int prefetch;           // slots are final before the kernels in front of this one end: fetch states early
};

// A warp owns the state rows warp, warp + 8, ...; a lane CV neighbouring columns of the CTA's 32 CV.
template <typename T, int NR, int CV>
__global__ void __launch_bounds__(kThreads, NR * CV <= 32 ? 2 : 1) ssd_step_kernel(StepArgs s) {
  constexpr int VS = 32 * CV;
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, sq_id = blockIdx.z, slice = blockIdx.x;
  const int per = a.heads / a.groups, hg = h / per, v0 = slice * VS, nv = min(VS, V - v0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c0 = lane * CV;
  const int n_in = 2 * D + nv;
  float* red = sm;                       // [2][8][VS]
  float* buf = red + 2 * 8 * VS;         // [2][2 D + VS]: B, C, x of a token
  float* wt = buf + 2 * (2 * D + VS);    // [2 D + VS][taps]: convolution weights
  float* wb = wt + (2 * D + VS) * a.taps;
  const int row0 = a.seq_row != nullptr ? a.seq_row[sq_id] : sq_id, len = a.seq_len != nullptr ? a.seq_len[sq_id] : 1;
  const int xc = h * V + v0, bc = a.heads * V + hg * D, cc = bc + a.groups * D;
  const bool col = c0 < nv;              // CV divides V: a lane's columns exist together
  auto channel = [&](int i) { return i < D ? bc + i : i < 2 * D ? cc + i - D : xc + i - 2 * D; };
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
  for (int i = tid; i < n_in; i += kThreads) {
    const int c = channel(i);
    for (int j = 0; j < a.taps; ++j) wt[i * a.taps + j] = DT<T>::to_f(reinterpret_cast<const T*>(a.conv)[(int64_t)c * a.taps + j]);
    wb[i] = a.conv_b[c];
  }
  const float rate = expf(a.a_log[h]), dtb = a.dt_bias[h], skip = a.skip[h];
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
  auto fetch = [&](int j) {              // token j of the sequence into its buffer
    float* b = buf + (j & 1) * (2 * D + VS);
    for (int i = tid; i < n_in; i += kThreads) {
      const float x = conv_silu<T>(a, channel(i), row0 + j, j, p0 + j, start, slot, wt + i * a.taps + a.taps - 1, wb[i]);
      b[i] = i < 2 * D ? x : rounded<T>(x);
    }
  };
  fetch(0);
  float z = a.dt[(int64_t)row0 * a.ldt + h];
  __syncthreads();
  for (int j = 0; j < len; ++j) {
    const float *B = buf + (j & 1) * (2 * D + VS), *C = B + D;
    float* rd = red + (j & 1) * (8 * VS);
    const float dt = softplusf(z + dtb), keep = expf(-rate * dt);
    float x[CV], w[CV], y[CV];
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      x[c] = col ? B[2 * D + c0 + c] : 0.f;
      w[c] = dt * x[c];
      y[c] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float bd = B[d], cd = C[d];
#pragma unroll
        for (int c = 0; c < CV; ++c) {
          S[i][c] = fmaf(bd, w[c], keep * S[i][c]);
          y[c] = fmaf(S[i][c], cd, y[c]);
        }
      }
    }
    store_cols<CV>(rd + warp * VS + c0, y);
    if (j + 1 < len) {
      z = a.dt[(int64_t)(row0 + j + 1) * a.ldt + h];
      fetch(j + 1);
    }
    __syncthreads();
    if (warp != (j & 7)) continue;       // the warps take turns with the sums
#pragma unroll
    for (int c = 0; c < CV; ++c) y[c] = skip * x[c];
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      float p[CV];
      load_cols<CV>(rd + q * VS + c0, p);
#pragma unroll
      for (int c = 0; c < CV; ++c) y[c] += p[c];
    }
    if (col) {
#pragma unroll
      for (int c = 0; c < CV; ++c) s.raw[((int64_t)(row0 + j) * a.heads + h) * V + v0 + c0 + c] = y[c];
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = warp + 8 * i;
    if (col && d < D) store_cols<CV>(st + (int64_t)d * V, S[i]);
  }
  if (s.ring_write) {
    // nobody reads this row in this launch; the first head of a group files the shared channels
    T* ring = reinterpret_cast<T*>(a.ring) + ((int64_t)slot * a.taps + p0 % a.taps) * a.channels;
    const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)row0 * a.ldp;
    for (int i = tid; i < n_in; i += kThreads) {
      if (i < 2 * D && (slice != 0 || h % per != 0)) continue;
      const int c = channel(i);
      ring[c] = proj[c];
    }
  }
}

// ---------------------------------------------------------------------------------------------- in chunks
// Scratch, laid out like the shared memory that reads it.  Of a (chunk, group): C and B of 32 rows, then their products.  Of
// a (chunk, head): P [32][36], read factors [32], write factors [32], the chunk's decay and the skip factor; then x [32][40]
// per slice of 32 columns.
struct Scratch {
  static constexpr int ldp = 36, ldv = 40;
  int Dp, slices, ld;
  __host__ __device__ Scratch(int D, int V)
      : Dp((D + 7) / 8 * 8), slices((V + kVS - 1) / kVS), ld(Dp % 16 == 0 ? Dp + 8 : Dp) {}
  __host__ __device__ int b() const { return kC * ld; }
  __host__ __device__ int cb() const { return 2 * kC * ld; }
  __host__ __device__ int group_floats() const { return cb() + kC * ldp; }
  __host__ __device__ int read() const { return kC * ldp; }
  __host__ __device__ int write() const { return read() + kC; }
  __host__ __device__ int ends() const { return write() + kC; }
  __host__ __device__ int head_part() const { return ends() + 4; }
  __host__ __device__ int x(int slice) const { return head_part() + slice * kC * ldv; }
  __host__ __device__ int head_floats() const { return x(slices); }
  // a stage: C, B | P and factors | x
  __host__ __device__ int stage() const { return cb() + head_part() + kC * ldv; }
};

struct ChunkArgs {
  Common c;
  const int* chunk_seq;     // [all chunks] sequence of a chunk
  const int* seq_chunk;     // [sequences + 1] first chunk of a sequence
  float* group_scratch;     // of the chunks [c0, c1), [chunk - c0][group]
  float* head_scratch;      // [chunk - c0][head]
  float* raw;               // y [tokens, heads, vdim]
  int* err;
  int c0, c1;
  int vec;                  // rows of proj and ring can be read 16 bytes at a time
};

// Convolution and silu of `width` neighbouring channels of a chunk from channel c0 on; put(token, channel - c0, n values).  ws:
// room for [taps][width] and a bias row.
template <typename T, int TP, typename F>
__device__ __forceinline__ void conv_chunk(const Common& a, bool vec, int c0, int width, int t0, int row0, int off, int p0,
                                           int start, int slot, int n, float* ws, F&& put) {
  const int tid = threadIdx.x;
  const T* w = reinterpret_cast<const T*>(a.conv) + (int64_t)c0 * a.taps;
  float* bs = ws + a.taps * width;
  const int nt = blockDim.x;
  for (int i = tid; i < width; i += nt) {
    for (int j = 0; j < a.taps; ++j) ws[j * width + i] = DT<T>::to_f(w[i * a.taps + j]);
    bs[i] = a.conv_b[c0 + i];
  }
  __syncthreads();
  if (vec) {
    const int nvec = width / 8;
    for (int i = tid; i < nvec * (kC / 4); i += nt) {
      const int c = (i % nvec) * 8, first = (i / nvec) * 4;
      float acc[4][8];
      conv_block<T, TP>(a, c0 + c, t0, row0, p0, start, slot, n, first, ws + c, width, acc, bs + c);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[j][e] = first + j < n ? fast_silu(acc[j][e]) : 0.f;
        put(first + j, c, acc[j], std::integral_constant<int, 8>{});
      }
    }
  } else {
    for (int i = tid; i < kC * width; i += nt) {
      const int t = i / width, c = i % width;
      const float v = t < n ? conv_silu<T>(a, c0 + c, t0 + t, off + t, p0 + t, start, slot, w + (int64_t)c * a.taps + a.taps - 1, bs[c])
                            : 0.f;
      put(t, c, &v, std::integral_constant<int, 1>{});
    }
  }
}

// n neighbouring values (n = 8: 16-byte aligned)
template <int N>
__device__ __forceinline__ void put_values(float* dst, const float* v) {
  if constexpr (N == 8) {
    *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(dst + 4) = make_float4(v[4], v[5], v[6], v[7]);
  } else {
    dst[0] = v[0];
  }
}

template <typename T, int TP>
__global__ void __launch_bounds__(kThreads) ssd_groups_kernel(ChunkArgs s) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, gi = blockIdx.y, chunk = s.c0 + blockIdx.x;
  const Scratch L(D, a.vdim);
  const int Dp = L.Dp, ld = Dp + 4;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* sB = sm;                        // [32][Dp + 4]
  float* sC = sB + kC * ld;
  float* ws = sC + kC * ld;              // [taps + 1][D]
  const int seq = s.chunk_seq[chunk], row0 = a.seq_row[seq], off = (chunk - s.seq_chunk[seq]) * kC;
  const int n = min(kC, a.seq_len[seq] - off), t0 = row0 + off;
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0] + off;
  float* out = s.group_scratch + ((int64_t)(chunk - s.c0) * a.groups + gi) * L.group_floats();
  const int bc = a.heads * a.vdim + gi * D;
  if (Dp > D)
    for (int i = tid; i < kC * (Dp - D); i += kThreads) {
      const int t = i / (Dp - D), d = D + i % (Dp - D);
      sB[t * ld + d] = sC[t * ld + d] = 0.f;
    }
  conv_chunk<T, TP>(a, s.vec != 0, bc, D, t0, row0, off, p0, start, slot, n, ws,
                    [&](int t, int c, const float* v, auto k) { put_values<decltype(k)::value>(sB + t * ld + c, v); });
  __syncthreads();
  conv_chunk<T, TP>(a, s.vec != 0, bc + a.groups * D, D, t0, row0, off, p0, start, slot, n, ws,
                    [&](int t, int c, const float* v, auto k) { put_values<decltype(k)::value>(sC + t * ld + c, v); });
  __syncthreads();
  for (int i = tid; i < kC * Dp; i += kThreads) {
    const int t = i / Dp, d = i % Dp;
    out[t * L.ld + d] = sC[t * ld + d];
    out[L.b() + t * L.ld + d] = sB[t * ld + d];
  }
  const int m0 = (warp >> 2) * 16, n0 = (warp & 3) * 8;
  Acc x;
  x.zero();
  if (n0 <= m0 + 15)
    for (int k0 = 0; k0 < Dp; k0 += 8)
      x.mac(frag_a([&](int r, int k) { return sC[(m0 + r) * ld + k0 + k]; }, g, t4),
            frag_b([&](int k, int j) { return sB[(n0 + j) * ld + k0 + k]; }, g, t4));
#pragma unroll
  for (int i = 0; i < 4; ++i) out[L.cb() + (m0 + g + 8 * (i >> 1)) * L.ldp + n0 + 2 * t4 + (i & 1)] = x.get(i);
}

// 64 to 256 threads
template <typename T, int TP>
__global__ void __launch_bounds__(kThreads) ssd_heads_kernel(ChunkArgs s) {
  extern __shared__ __align__(16) float sm[];      // [taps + 1][vdim] convolution weights
  // running sum of the decays' logarithms, in 64-bit: its differences must keep 32-bit accuracy when single tokens decay
  // to nothing
  __shared__ double sL[kC];
  __shared__ float sD[kC];
  const Common& a = s.c;
  const int V = a.vdim, h = blockIdx.y, chunk = s.c0 + blockIdx.x, gi = h / (a.heads / a.groups);
  const Scratch L(a.dim, V);
  const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31;
  const int seq = s.chunk_seq[chunk], row0 = a.seq_row[seq], off = (chunk - s.seq_chunk[seq]) * kC;
  const int n = min(kC, a.seq_len[seq] - off), t0 = row0 + off;
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0] + off;
  float* out = s.head_scratch + ((int64_t)(chunk - s.c0) * a.heads + h) * L.head_floats();
  const float* cb = s.group_scratch + ((int64_t)(chunk - s.c0) * a.groups + gi) * L.group_floats() + L.cb();
  if (tid < 32) {
    double lg = 0.0;
    float dt = 0.f;
    if (lane < n) {
      dt = softplusf(a.dt[(int64_t)(t0 + lane) * a.ldt + h] + a.dt_bias[h]);
      lg = -(double)(expf(a.a_log[h]) * dt);
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double x = __shfl_up_sync(0xffffffffu, lg, o);
      if (lane >= o) lg += x;
    }
    const double end = __shfl_sync(0xffffffffu, lg, 31);
    sL[lane] = lg;
    sD[lane] = dt;
    out[L.read() + lane] = expf((float)lg);
    out[L.write() + lane] = dt * expf((float)(end - lg));
    if (lane < 4) out[L.ends() + lane] = lane == 0 ? expf((float)end) : lane == 1 ? a.skip[h] : 0.f;
  }
  const int Vp = L.slices * kVS;
  if (Vp > V)
    for (int i = tid; i < kC * (Vp - V); i += nt) {
      const int t = i / (Vp - V), c = V + i % (Vp - V);
      out[L.x(c / kVS) + t * L.ldv + c % kVS] = 0.f;
    }
  conv_chunk<T, TP>(a, s.vec != 0, h * V, V, t0, row0, off, p0, start, slot, n, sm, [&](int t, int c, const float* v, auto k) {
    constexpr int N = decltype(k)::value;
    float x[N];
#pragma unroll
    for (int e = 0; e < N; ++e) x[e] = rounded<T>(v[e]);
    put_values<N>(out + L.x(c / kVS) + t * L.ldv + c % kVS, x);
  });
  // (conv_chunk's barrier: the sums are in place)
  for (int i = tid; i < kC * kC; i += nt) {
    const int t = i >> 5, j = i & 31;
    out[t * L.ldp + j] = j <= t ? cb[t * L.ldp + j] * sD[j] * expf((float)(sL[t] - sL[j])) : 0.f;
  }
}

size_t groups_smem(const Scratch& L, int D, int taps) {
  return ((size_t)2 * kC * (L.Dp + 4) + (size_t)(taps + 1) * D) * sizeof(float);
}
size_t chunk_smem(const Scratch& L, int stages) {
  return ((size_t)stages * L.stage() + 4 * kC * 36) * sizeof(float);
}

// CTA = 32 state columns of one head of one sequence.  Warp (vt, dg): columns 16 vt .. + 15, channel tiles of share dg; S^T
// in accumulator fragments.  The four shares' read-outs meet in shared memory.
template <int MT, int PER_SM>
__global__ void __launch_bounds__(kThreads, PER_SM) ssd_chunks_kernel(ChunkArgs s, int stages) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(8) uint64_t full[4];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kVS, nv = min(kVS, V - v0);
  const int gi = h / (a.heads / a.groups);
  const Scratch L(D, V);
  const int Dp = L.Dp, ld = L.ld, tiles = Dp / 8, per = (tiles + 3) / 4;
  const int first = s.seq_chunk[seq], last = s.seq_chunk[seq + 1];
  const int ca = max(first, s.c0), cb = min(last, s.c1);
  if (ca >= cb) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int vt = warp & 1, dg = warp >> 1;
  float* red = sm + stages * L.stage();        // [4][32][36]
  const int row0 = a.seq_row[seq], len = a.seq_len[seq];
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0;
  auto fetch = [&](int c) {                    // one thread
    if (c >= cb) return;
    const float* gs = s.group_scratch + ((int64_t)(c - s.c0) * a.groups + gi) * L.group_floats();
    const float* hs = s.head_scratch + ((int64_t)(c - s.c0) * a.heads + h) * L.head_floats();
    float* dst = sm + ((c - ca) % stages) * L.stage();
    uint64_t* bar = &full[(c - ca) % stages];
    tc5::mbar_expect_tx(bar, (uint32_t)(L.stage() * sizeof(float)));
    bulk_load(dst, gs, (uint32_t)(L.cb() * sizeof(float)), bar);
    bulk_load(dst + L.cb(), hs, (uint32_t)(L.head_part() * sizeof(float)), bar);
    bulk_load(dst + L.cb() + L.head_part(), hs + L.x(blockIdx.x), (uint32_t)(kC * L.ldv * sizeof(float)), bar);
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
      if (lane == 0) tc5::report(s.err, 43);
      ok = false;
    }
    const float* Q = sm + (at % stages) * L.stage();
    const float *K = Q + L.b(), *P = Q + L.cb(), *X = P + L.head_part(), *Xw = X + vt * 16;
    if (ok) {
      const float *rf = P + L.read(), *wf = P + L.write();
      // ---- O^T = S^T C^T: the state's fragments are the left operand (k order inside a tile: 0 2 4 6 1 3 5 7)
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
      // ---- ... times the tokens' read factors
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const float2 f = *reinterpret_cast<const float2*>(rf + n * 8 + 2 * t4);
        o[n][0] *= f.x;
        o[n][1] *= f.y;
        o[n][2] *= f.x;
        o[n][3] *= f.y;
      }
      // x as left operand, exact in one part
      uint32_t va[4][4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float* v = Xw + (k * 8 + t4) * L.ldv + g;
        va[k][0] = __float_as_uint(v[0]);
        va[k][1] = __float_as_uint(v[8]);
        va[k][2] = __float_as_uint(v[4 * L.ldv]);
        va[k][3] = __float_as_uint(v[4 * L.ldv + 8]);
      }
      // ---- ... + X^T P^T, this warp's eight keys
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (k == dg) {
#pragma unroll
          for (int n = 0; n < 4; ++n)
            if (n >= k) mac2(o[n], va[k], frag_b([&](int kk, int j) { return P[(n * 8 + j) * L.ldp + k * 8 + kk]; }, g, t4));
        }
      float* rd = red + dg * (kC * 36) + vt * 16;
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) rd[(n * 8 + 2 * t4 + (i & 1)) * 36 + g + 8 * (i >> 1)] = o[n][i];
      // ---- S^T <- S^T decay + X^T (f B)
      const int mine = min(per, tiles - dg * per);       // tiles of this warp that exist
      float add[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i) add[m][i] = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float f0 = wf[k * 8 + t4], f1 = wf[k * 8 + t4 + 4];
        FragB fb[MT];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < mine)
            fb[m] = frag_b([&](int kk, int j) { return K[(k * 8 + kk) * ld + (dg * per + m) * 8 + j] * (kk < 4 ? f0 : f1); }, g, t4);
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < mine) mma_tf32(add[m], va[k], fb[m].lo);
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < mine) mma_tf32(add[m], va[k], fb[m].hi);
      }
      const float keep = P[L.ends()];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        if (m < mine) {
#pragma unroll
          for (int i = 0; i < 4; ++i) S[m][i] = fmaf(keep, S[m][i], add[m][i]);
        }
    }
    // what the sums below need of this stage
    const float skip = ok ? P[L.ends() + 1] : 0.f;
    float xs[kC * kVS / kThreads];
#pragma unroll
    for (int i = 0; i < kC * kVS / kThreads; ++i) xs[i] = ok ? X[(warp + 8 * i) * L.ldv + lane] : 0.f;
    if (__syncthreads_or(!ok)) {               // the parts are in place, the stage is free again
      ok = false;
      break;
    }
    if (tid == 0) fetch(c + stages);
    const int off = (c - first) * kC;
    const float* rd = red;
#pragma unroll
    for (int i = 0; i < kC * kVS / kThreads; ++i) {
      const int t = warp + 8 * i;
      const float y = (rd[t * 36 + lane] + rd[(kC + t) * 36 + lane]) +
                      (rd[(2 * kC + t) * 36 + lane] + rd[(3 * kC + t) * 36 + lane]);
      if (off + t < len && lane < nv) s.raw[((int64_t)(row0 + off + t) * a.heads + h) * V + v0 + lane] = fmaf(skip, xs[i], y);
    }
    __syncthreads();                           // the sums are read
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

bool sizes_ok(int heads, int groups, int dim, int vdim, int taps) {
  return heads >= 1 && heads <= 65535 && groups >= 1 && heads % groups == 0 && dim >= 1 && dim <= 512 && vdim >= 1 &&
         vdim <= 65535 && taps >= 1;
}

template <typename T, int NR, int CV>
cudaError_t launch_step(const StepArgs& s, int seqs, bool pdl, cudaStream_t st) {
  const int slices = (s.c.vdim + 32 * CV - 1) / (32 * CV);
  const size_t smem = ((3 + (size_t)s.c.taps) * (2 * (size_t)s.c.dim + 32 * CV) + 2 * 8 * 32 * CV) * sizeof(float);
  if (smem > kSmemMax) return cudaErrorInvalidValue;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(ssd_step_kernel<T, NR, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_kernel(ssd_step_kernel<T, NR, CV>, dim3(slices, s.c.heads, seqs), dim3(kThreads), smem, st, pdl, s);
}

// Columns per lane: as many as V divides into and the registers of NR rows leave room for, fewer while that spreads the
// large states of a few sequences over more SMs.
template <typename T, int NR>
cudaError_t pick_cols(const StepArgs& s, int seqs, bool pdl, cudaStream_t st) {
  const int V = s.c.vdim;
  int cv = NR <= 16 && V % 4 == 0 && V > 64 ? 4 : NR <= 32 && V % 2 == 0 && V > 32 ? 2 : 1;
  while (cv > 1 && s.c.dim * 32 * cv > 4096 && (int64_t)s.c.heads * seqs * ((V + 16 * cv - 1) / (16 * cv)) <= 2 * 148) cv /= 2;
  if constexpr (NR <= 16)
    if (cv == 4) return launch_step<T, NR, 4>(s, seqs, pdl, st);
  if constexpr (NR <= 32)
    if (cv == 2) return launch_step<T, NR, 2>(s, seqs, pdl, st);
  return launch_step<T, NR, 1>(s, seqs, pdl, st);
}

Common common_args(const void* proj, int64_t ldp, const float* dt, int64_t ldt, const void* conv, const float* conv_b,
                   const float* dt_bias, const float* a_log, const float* skip, void* ring, float* state, const int* slot,
                   const int* pos, const int* start, const int* seq_row, const int* seq_len, int heads, int groups, int dim,
                   int vdim, int taps) {
  return Common{proj, dt, conv, conv_b, dt_bias, a_log, skip, ring, state, slot, pos, start, seq_row, seq_len, ldp, ldt,
                heads, groups, dim, vdim, taps, heads * vdim + 2 * groups * dim};
}

}  // namespace

// Can the chunked form take these sizes?
IPEX_API int ipex_ssd_chunks_ok(int dim, int vdim, int taps) {
  const Scratch L(dim, vdim);
  return dim >= 1 && dim <= 256 && vdim >= 1 && taps >= 1 && groups_smem(L, dim, taps) <= kSmemMax &&
         (size_t)(taps + 1) * vdim * sizeof(float) <= kSmemMax - 1024 && chunk_smem(L, 1) <= kSmemMax;
}
IPEX_API int64_t ipex_ssd_group_floats(int dim, int vdim) { return Scratch(dim, vdim).group_floats(); }
IPEX_API int64_t ipex_ssd_head_floats(int dim, int vdim) { return Scratch(dim, vdim).head_floats(); }

// Token by token.  seq_row / seq_len null: `seqs` sequences of one token each, whose convolution inputs are filed on the
// way.  raw [tokens, heads, vdim]: the outputs.
IPEX_API int ipex_ssd_step(const void* proj, int64_t ldp, const float* dt, int64_t ldt, const void* conv, const float* conv_b,
                           const float* dt_bias, const float* a_log, const float* skip, void* ring, float* state,
                           const int* slot, const int* pos, const int* start, const int* seq_row, const int* seq_len, int seqs,
                           float* raw, int heads, int groups, int dim, int vdim, int taps, int dtype, int pdl, void* stream) {
  if (!sizes_ok(heads, groups, dim, vdim, taps) || seqs < 1 || seqs > 65535 || (seq_row == nullptr) != (seq_len == nullptr) ||
      raw == nullptr)
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    StepArgs s = {common_args(proj, ldp, dt, ldt, conv, conv_b, dt_bias, a_log, skip, ring, state, slot, pos, start, seq_row,
                              seq_len, heads, groups, dim, vdim, taps),
                  raw, seq_row == nullptr, pdl && seq_row == nullptr && vdim % 4 == 0};
    cudaStream_t st = (cudaStream_t)stream;
    if (dim <= 32) return pick_cols<T, 4>(s, seqs, pdl != 0, st);
    if (dim <= 64) return pick_cols<T, 8>(s, seqs, pdl != 0, st);
    if (dim <= 128) return pick_cols<T, 16>(s, seqs, pdl != 0, st);
    if (dim <= 256) return pick_cols<T, 32>(s, seqs, pdl != 0, st);
    return pick_cols<T, 64>(s, seqs, pdl != 0, st);
  });
}

// Chunks [c0, c1) of a packed batch in the chunked form (16-bit models).  chunk_seq [chunks], seq_chunk [seqs + 1]: device
// tables of the sequences' chunks of 32 tokens, in order; scratch: (c1 - c0) * groups * ipex_ssd_group_floats and (c1 - c0) *
// heads * ipex_ssd_head_floats; raw as above.  The ring is read, not written (ipex_ring_tail).
IPEX_API int ipex_ssd_chunks(const void* proj, int64_t ldp, const float* dt, int64_t ldt, const void* conv,
                             const float* conv_b, const float* dt_bias, const float* a_log, const float* skip, void* ring,
                             float* state, const int* slot, const int* pos, const int* start, const int* seq_row,
                             const int* seq_len, int seqs, const int* chunk_seq, const int* seq_chunk, int c0, int c1,
                             float* group_scratch, float* head_scratch, float* raw, int heads, int groups, int dim, int vdim,
                             int taps, int dtype, int* err, void* stream) {
  if (!sizes_ok(heads, groups, dim, vdim, taps) || !ipex_ssd_chunks_ok(dim, vdim, taps) || seqs < 1 || seqs > 65535 ||
      c0 < 0 || c1 <= c0 || seq_row == nullptr || seq_len == nullptr ||
      (((uintptr_t)group_scratch | (uintptr_t)head_scratch) & 15) || dtype == DT_F32)
    return (int)cudaErrorInvalidValue;
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ChunkArgs s = {common_args(proj, ldp, dt, ldt, conv, conv_b, dt_bias, a_log, skip, ring, state, slot, pos, start, seq_row,
                               seq_len, heads, groups, dim, vdim, taps),
                   chunk_seq, seq_chunk, group_scratch, head_scratch, raw, err, c0, c1, 0};
    s.vec = dim % 8 == 0 && vdim % 8 == 0 && ldp % 8 == 0 && (((uintptr_t)proj | (uintptr_t)ring) & 15) == 0;
    cudaStream_t st = (cudaStream_t)stream;
    const Scratch L(dim, vdim);
    const size_t gs = groups_smem(L, dim, taps), hs = (size_t)(taps + 1) * vdim * sizeof(float);
    auto prep_g = taps == 4 ? ssd_groups_kernel<T, 4> : ssd_groups_kernel<T, 0>;
    auto prep_h = taps == 4 ? ssd_heads_kernel<T, 4> : ssd_heads_kernel<T, 0>;
    cudaError_t e = cudaFuncSetAttribute(prep_g, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gs);
    if (e == cudaSuccess && hs > 40 * 1024) e = cudaFuncSetAttribute(prep_h, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)hs);
    if (e != cudaSuccess) return e;
    prep_g<<<dim3(c1 - c0, groups), kThreads, gs, st>>>(s);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const int items = vdim / 8 * (kC / 4), ht = items <= 64 ? 64 : items <= 128 ? 128 : kThreads;
    prep_h<<<dim3(c1 - c0, heads), ht, hs, st>>>(s);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    // more CTAs than SMs: two per SM with fewer stages each
    const bool pairs = dim <= 128 && (int64_t)L.slices * heads * seqs > 148;
    int stages = 4;
    while (stages > 1 && chunk_smem(L, stages) > (pairs ? kSmemMax / 2 : kSmemMax)) --stages;
    const size_t cs = chunk_smem(L, stages);
    auto kern = dim <= 64    ? (pairs ? ssd_chunks_kernel<2, 2> : ssd_chunks_kernel<2, 1>)
                : dim <= 128 ? (pairs ? ssd_chunks_kernel<4, 2> : ssd_chunks_kernel<4, 1>)
                             : ssd_chunks_kernel<8, 1>;
    e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cs);
    if (e != cudaSuccess) return e;
    kern<<<dim3(L.slices, heads, seqs), kThreads, cs, st>>>(s, stages);
    return cudaGetLastError();
  };
  return (int)(dtype == DT_F16 ? run((__half*)nullptr) : run((__nv_bfloat16*)nullptr));
}
