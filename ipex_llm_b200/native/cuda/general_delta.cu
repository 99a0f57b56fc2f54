// Generalized delta rule with decays and removal rates per key channel, sm_100a.
//
// Per head a matrix state S [dim, vdim] is carried from token to token:
//     S <- diag(w) S - (a * u) (u^T S) + k v^T;   o = S^T r          u = k / |k|, both terms read the old state
//     w = exp(-c sigmoid(z)),  z = up . tanh(low) + bias;            a = sigmoid(rate + rate_bias)
// r, k, v and the rates come from projections; z from a low-rank pair whose first half (`low`) is a projection too.
// z, w, a, u, the state and the products that touch it are fp32.
//
//   general_step    token by token, state in registers: decoding (one token of every sequence; the gated norm of the
//                   output is fused), short portions, 32-bit models
//   general_prep    prompts, first half, parallel over chunks of 32 tokens (below)
//   general_chunks  second half, sequential over a sequence's chunks:
//                   X = W S, O = Ob + Q' S, S <- diag(L_end) S + U - B^T X
//
// With L_t the product of the decays inside a chunk, up to and with token t:  p_t = L_(t-1) u_t,  q_t = L_t r_t,
// b_t = a_t u_t / L_t,  g_t = k_t / L_t.  What token t reads of the old state is y_t = S_(t-1)^T u_t, and
//     (I + A) Y = P S + M V,   A[t,i] = p_t . b_i, M[t,i] = p_t . g_i for i < t;    T = (I + A)^-1
//     O = Q S + E V - H Y,     E[t,i] = q_t . g_i, H[t,i] = q_t . b_i for i <= t
//     S_end = diag(L_end) (S + g^T V - b^T Y)
// so the half that runs in parallel leaves  W = T P,  Q' = Q - H W,  Ob = (E - H T M) V,  B = b L_end and
// U = (g L_end - (T M)^T B)^T V.  A decay is never below exp(-c), which bounds 1 / L (the launch checks c): the quotients
// keep their relative accuracy and every product of two of them is again a product of decays.
//
// Products of the chunked form run on the tensor cores with fp32 operands split into tf32 pairs (values as they come from
// a 16-bit projection need one part only).  The state's columns are independent, so a head is spread over slices of 32.
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
constexpr float kUnitEps = 1e-6f;
constexpr float kMaxLog = 64.f;       // most that a chunk's decays may add up to in the chunked form

template <typename F>
int by_dtype(int dtype, F&& f) {
  if (dtype == DT_F16) return (int)f((__half*)nullptr);
  if (dtype == DT_BF16) return (int)f((__nv_bfloat16*)nullptr);
  if (dtype == DT_F32) return (int)f((float*)nullptr);
  return (int)cudaErrorInvalidValue;
}

struct Common {
  const void* proj;       // T [tokens, ldp]: r heads, k heads, v heads, rates, output gates
  const float* low;       // [tokens, ldl], the first `rank` columns
  const void* up;         // T [heads * dim, rank]
  const float* bias;      // [heads * dim]
  const float* rate_bias; // [heads * dim]
  float* state;           // [slots, heads, dim, vdim]
  const int* slot;        // [tokens]
  const int* pos;         // [tokens]
  const int* start;       // [slots]
  const int* seq_row;     // [sequences] first packed token, or null: sequence = token
  const int* seq_len;
  int64_t ldp, ldl;
  int heads, dim, vdim, rank;
  float c;                // decays are exp(-c sigmoid(z))
};

// ---------------------------------------------------------------------------------------------- token by token
struct StepArgs {
  Common c;
  const void* norm_w;     // fused norm (one token per sequence): T [heads * vdim], out T [tokens, ldo]
  void* out;
  float* raw;             // else: o [tokens, heads, vdim]
  int64_t ldo;
  float eps;
  int gate_off;           // column of the output gates in proj
  int prefetch;           // slots are final before the kernels in front of this one end: fetch states early
  int staged;             // the head's rows of `up` fit shared memory
};

// A warp owns the state rows warp, warp + 8, ...; a lane CV neighbouring columns of the CTA's 32 CV.
template <typename T, int NR, int CV>
__global__ void __launch_bounds__(kThreads, NR * CV <= 64 ? 2 : 1) general_step_kernel(StepArgs s) {
  constexpr int VS = 32 * CV;
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, sq_id = blockIdx.z, slice = blockIdx.x;
  const int v0 = slice * VS, nv = min(VS, V - v0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c0 = lane * CV;
  const int ldb = 4 * D + VS, ldr = a.rank | 1;
  float* red = sm;                      // [2][2][8][VS]
  float* buf = red + 2 * 2 * 8 * VS;    // [2][4 D + VS]: r, k, decay, rate, v of a token
  float* slow = buf + 2 * ldb;          // [2][rank]: tanh(low) of a token
  float* sup = slow + 2 * a.rank;       // [D][rank | 1]
  __shared__ float s_ss;
  const int row0 = a.seq_row != nullptr ? a.seq_row[sq_id] : sq_id, len = a.seq_len != nullptr ? a.seq_len[sq_id] : 1;
  const int rc = h * D, kc = a.heads * D + rc, vc = 2 * a.heads * D + h * V + v0, ac = a.heads * (2 * D + V) + rc;
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
  const float *bias = a.bias + h * D, *rbias = a.rate_bias + h * D;
  if (s.staged)
    for (int i = tid; i < D * a.rank; i += kThreads) sup[i / a.rank * ldr + i % a.rank] = DT<T>::to_f(up[i]);
  float nw[CV];
#pragma unroll
  for (int c = 0; c < CV; ++c)
    nw[c] = s.raw == nullptr && col ? DT<T>::to_f(reinterpret_cast<const T*>(s.norm_w)[h * V + v0 + c0 + c]) : 0.f;
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
  auto stage_low = [&](int j) {
    if (j < len)
      for (int i = tid; i < a.rank; i += kThreads) slow[(j & 1) * a.rank + i] = tanhf(a.low[(int64_t)(row0 + j) * a.ldl + i]);
  };
  auto fetch = [&](int j) {             // token j of the sequence into its buffer
    const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)(row0 + j) * a.ldp;
    const float* low = slow + (j & 1) * a.rank;
    float* b = buf + (j & 1) * ldb;
    for (int i = tid; i < 4 * D + nv; i += kThreads) {
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
        b[2 * D + i] = expf(-a.c * sigmoidf(z0 + z1));
      } else if (i < 2 * D) {
        b[i - D] = DT<T>::to_f(proj[rc + i - D]);
      } else if (i < 3 * D) {
        b[i - D] = DT<T>::to_f(proj[kc + i - 2 * D]);
      } else if (i < 4 * D) {
        b[i] = sigmoidf(DT<T>::to_f(proj[ac + i - 3 * D]) + rbias[i - 3 * D]);
      } else {
        b[i] = DT<T>::to_f(proj[vc + i - 4 * D]);
      }
    }
  };
  float gate[CV];
  if (s.raw == nullptr && warp == 0 && col) {
#pragma unroll
    for (int c = 0; c < CV; ++c)
      gate[c] = DT<T>::to_f(reinterpret_cast<const T*>(a.proj)[(int64_t)row0 * a.ldp + s.gate_off + h * V + v0 + c0 + c]);
  }
  stage_low(0);
  __syncthreads();                      // (and `sup`)
  fetch(0);
  stage_low(1);
  __syncthreads();
  for (int j = 0; j < len; ++j) {
    const float* b = buf + (j & 1) * ldb;
    const float *r = b, *k = b + D, *w = b + 2 * D, *rate = b + 3 * D;
    float* rd = red + (j & 1) * (2 * 8 * VS);
    float kk = 0.f, rk = 0.f, ra = 0.f;
    for (int d = lane; d < D; d += 32) {
      kk = fmaf(k[d], k[d], kk);
      rk = fmaf(r[d], k[d], rk);
      ra = fmaf(r[d] * rate[d], k[d], ra);
    }
    float sk[CV], sr[CV];
#pragma unroll
    for (int c = 0; c < CV; ++c) sk[c] = sr[c] = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float kd = k[d], wr = w[d] * r[d];
#pragma unroll
        for (int c = 0; c < CV; ++c) {
          sk[c] = fmaf(S[i][c], kd, sk[c]);
          sr[c] = fmaf(S[i][c], wr, sr[c]);
        }
      }
    }
    store_cols<CV>(rd + warp * VS + c0, sk);
    store_cols<CV>(rd + (8 + warp) * VS + c0, sr);
    const float ik = 1.0f / sqrtf(warp_sum(kk) + kUnitEps);
    rk = warp_sum(rk);
    ra = warp_sum(ra) * ik;
    __syncthreads();
#pragma unroll
    for (int c = 0; c < CV; ++c) sk[c] = sr[c] = 0.f;
#pragma unroll
    for (int wi = 0; wi < 8; ++wi) {
      float x[CV], y[CV];
      load_cols<CV>(rd + wi * VS + c0, x);
      load_cols<CV>(rd + (8 + wi) * VS + c0, y);
#pragma unroll
      for (int c = 0; c < CV; ++c) {
        sk[c] += x[c];
        sr[c] += y[c];
      }
    }
    float v[CV], y[CV], o[CV];
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      v[c] = col ? b[4 * D + c0 + c] : 0.f;
      const float seen = ik * sk[c];                   // u^T S of the old state
      o[c] = sr[c] + (rk * v[c] - ra * seen);          // S^T r after the write
      y[c] = ik * seen;
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float kd = k[d], wd = w[d], ad = rate[d];
#pragma unroll
        for (int c = 0; c < CV; ++c) S[i][c] = fmaf(kd, fmaf(-ad, y[c], v[c]), wd * S[i][c]);
      }
    }
    if (s.raw != nullptr) {
      if (warp == (j & 7) && col) {
#pragma unroll
        for (int c = 0; c < CV; ++c) s.raw[((int64_t)(row0 + j) * a.heads + h) * V + v0 + c0 + c] = o[c];
      }
      if (j + 1 < len) {
        fetch(j + 1);
        stage_low(j + 2);
        __syncthreads();
      }
    } else {
      // one token: norm over all columns of the head, which the CTAs of the cluster hold slice by slice
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < CV; ++c) ss = fmaf(o[c], o[c], ss);
      float total = ss = warp_sum(col ? ss : 0.f);
      if (gridDim.x > 1) {
        if (tid == 0) s_ss = ss;
        cg::cluster_group cluster = cg::this_cluster();
        cluster.sync();
        total = 0.f;
        for (int q = 0; q < (int)gridDim.x; ++q) total += *cluster.map_shared_rank(&s_ss, q);
        cluster.sync();
      }
      if (warp == 0 && col) {
        const float inv = 1.0f / sqrtf(total / (float)V + s.eps);
        T* out = reinterpret_cast<T*>(s.out) + (int64_t)row0 * s.ldo + h * V + v0 + c0;
#pragma unroll
        for (int c = 0; c < CV; ++c) out[c] = DT<T>::from_f(o[c] * inv * nw[c] * sigmoidf(gate[c]));
      }
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
// apart): W, Q' and B of 32 rows, decays of the whole chunk; then per slice of 32 columns Ob [32][40] and U [Dm][40].
struct Scratch {
  static constexpr int ldu = 40;
  int Dp, Dm, slices, ldw, ldk;
  __host__ __device__ Scratch(int D, int V)
      : Dp((D + 7) / 8 * 8), Dm((D + 15) / 16 * 16), slices((V + kVS - 1) / kVS), ldw(Dp + 4), ldk(Dp % 16 == 0 ? Dp + 8 : Dp) {}
  __host__ __device__ int q() const { return kC * ldw; }
  __host__ __device__ int b() const { return 2 * kC * ldw; }
  __host__ __device__ int g() const { return b() + kC * ldk; }
  __host__ __device__ int shared_part() const { return g() + Dm; }
  __host__ __device__ int slice_part() const { return (kC + Dm) * ldu; }
  __host__ __device__ int slice(int i) const { return shared_part() + i * slice_part(); }
  __host__ __device__ int floats() const { return slice(slices); }
  __host__ __device__ int stage() const { return shared_part() + slice_part(); }
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

constexpr int kLdM = 36;      // row stride of the 32 x 32 matrices
constexpr int kR = 64;        // columns of the decays' projection at a time
// Shared memory of general_prep: four arrays of 32 rows; what the decays' projection needs, later the 32 x 32 matrices; sums.
struct PrepLayout {
  int ld, ldv, ldu, lds;      // row strides: the arrays, v (in T), up (in T), low
  int mats, tot, floats;
  __host__ __device__ PrepLayout(const Scratch& L)
      : ld(L.Dp + 4), ldv(L.slices * kVS + 8), ldu(kR + 8), lds(kR + 4) {
    mats = 4 * kC * ld + kC * ldv / 2;
    const int proj = L.Dp * ldu / 2 + kC * lds, matrices = 7 * kC * kLdM;
    tot = mats + (proj > matrices ? proj : matrices);
    floats = tot + 4 * (L.Dp + 1) + kC;
  }
};
size_t prep_smem(const Scratch& L) { return (size_t)PrepLayout(L).floats * sizeof(float); }
size_t chunk_smem(const Scratch& L, int stages) {
  return ((size_t)(L.Dm + kC) * L.ldu + (size_t)stages * L.stage()) * sizeof(float);
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(tc5::smem_u32(dst)), "l"(src) : "memory");
}

// NZ: 64-channel tiles of a head.
template <typename T, int NZ>
__global__ void __launch_bounds__(kThreads, NZ == 1 ? 3 : NZ == 2 ? 2 : 1) general_prep_kernel(ChunkArgs s) {
  extern __shared__ __align__(16) float sm[];
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, chunk = s.c0 + blockIdx.x, rank = a.rank;
  const Scratch L(D, V);
  const PrepLayout PL(L);
  const int Dp = L.Dp, Vp = L.slices * kVS, ld = PL.ld, ldv = PL.ldv;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* sq = sm;                        // [32][Dp + 4]: r, then q
  float* sk = sq + kC * ld;              // k, then g
  float* sp = sk + kC * ld;              // running sum of the decays' logarithms, then p
  float* sb = sp + kC * ld;              // rates, then b
  T* sv = reinterpret_cast<T*>(sb + kC * ld);                // [32][Vp + 8]
  float* mA = sm + PL.mats;              // 32 x 32 matrices
  float* mM = mA + kC * kLdM;
  float* mE = mM + kC * kLdM;
  float* mH = mE + kC * kLdM;
  float* mT = mH + kC * kLdM;
  float* mTM = mT + kC * kLdM;
  float* mHT = mTM + kC * kLdM;
  T* sup = reinterpret_cast<T*>(mA);     // before them: [Dp][kR + 8] of `up`, ...
  float* slow = mA + L.Dp * PL.ldu / 2;  // ... [32][kR + 4] of tanh(low)
  float* tot = sm + PL.tot;              // [4][Dp + 1]: logarithms of eight tokens' decays
  float* sik = tot + 4 * (Dp + 1);       // [32] 1 / |k|
  const int seq = s.chunk_seq[chunk], row0 = a.seq_row[seq], off = (chunk - s.seq_chunk[seq]) * kC;
  const int n = min(kC, a.seq_len[seq] - off), t0 = row0 + off;
  float* out = s.scratch + ((int64_t)(chunk - s.c0) * a.heads + h) * L.floats();
  const T* proj = reinterpret_cast<const T*>(a.proj) + (int64_t)t0 * a.ldp;
  const int rc = h * D, kcol = a.heads * D + rc, vcol = 2 * a.heads * D + h * V, acol = a.heads * (2 * D + V) + rc;
  const bool vec = D % 8 == 0 && V % 8 == 0 && a.ldp % 8 == 0 && (reinterpret_cast<uintptr_t>(a.proj) & 15) == 0;

  // ---- operands (zeros behind the sequence's end and past the sizes): the first loads are in flight during the projection
  constexpr int kEarly = NZ <= 2 ? 4 * NZ : 8;
  const int nd = D / 8, per = 3 * nd + Vp / 8;
  uint4 early[kEarly];
  auto fetch = [&](int i) {
    const int t = i / per, c = i % per, what = min(c / max(nd, 1), 3), e0 = (c - what * nd) * 8;
    uint4 raw = make_uint4(0, 0, 0, 0);
    if (i < kC * per && t < n && (what < 3 || e0 < V))
      raw = *reinterpret_cast<const uint4*>(proj + (int64_t)t * a.ldp +
                                            (what == 0 ? rc : what == 1 ? kcol : what == 2 ? acol : vcol) + e0);
    return raw;
  };
  auto file = [&](int i, const uint4& raw) {
    if (i >= kC * per) return;
    const int t = i / per, c = i % per, what = min(c / nd, 3), e0 = (c - what * nd) * 8;
    if (what == 3) {
      *reinterpret_cast<uint4*>(sv + t * ldv + e0) = raw;
      return;
    }
    const T* e = reinterpret_cast<const T*>(&raw);
    float* dst = (what == 0 ? sq : what == 1 ? sk : sb) + t * ld + e0;
    float x[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] = DT<T>::to_f(e[j]);
    if (what == 2) {
      const float4 b0 = *reinterpret_cast<const float4*>(a.rate_bias + rc + e0);
      const float4 b1 = *reinterpret_cast<const float4*>(a.rate_bias + rc + e0 + 4);
      const float b[8] = {b0.x, b0.y, b0.z, b0.w, b1.x, b1.y, b1.z, b1.w};
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = t < n ? sigmoidf(x[j] + b[j]) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4*>(dst + j) = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
  };
  if (vec) {
#pragma unroll
    for (int u = 0; u < kEarly; ++u) early[u] = fetch(tid + u * kThreads);
  }
  // ---- z = up tanh(low): `up` is exact in one tf32 part; a warp has every eighth tile of eight channels, both row tiles
  float z[NZ][2][4];
#pragma unroll
  for (int j = 0; j < NZ; ++j)
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int i = 0; i < 4; ++i) z[j][m][i] = 0.f;
  const T* up = reinterpret_cast<const T*>(a.up) + (int64_t)h * D * rank;
  for (int r0 = 0; r0 < rank; r0 += kR) {
    const int nr = min(kR, rank - r0), nk = (nr + 7) / 8 * 8;
    if (r0 > 0) __syncthreads();
    if (rank % 8 == 0 && (reinterpret_cast<uintptr_t>(up) & 15) == 0) {
      const int nv = nk / 8;
      for (int i = tid; i < D * nv; i += kThreads) {
        const int d = i / nv, c = (i - d * nv) * 8;
        cp_async16(sup + d * PL.ldu + c, up + (int64_t)d * rank + r0 + c);
      }
      for (int i = D * nk + tid; i < Dp * nk; i += kThreads) sup[i / nk * PL.ldu + i % nk] = DT<T>::from_f(0.f);
    } else {
      for (int i = tid; i < Dp * nk; i += kThreads) {
        const int d = i / nk, c = i - d * nk;
        sup[d * PL.ldu + c] = d < D && c < nr ? up[(int64_t)d * rank + r0 + c] : DT<T>::from_f(0.f);
      }
    }
    for (int i = tid; i < kC * nk; i += kThreads) {
      const int t = i / nk, c = i - t * nk;
      slow[t * PL.lds + c] = t < n && c < nr ? tanhf(a.low[(int64_t)(t0 + t) * a.ldl + r0 + c]) : 0.f;
    }
    asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int k0 = 0; k0 < nk; k0 += 8) {
      FragA fa[2];
#pragma unroll
      for (int m = 0; m < 2; ++m) fa[m] = frag_a([&](int r, int k) { return slow[(m * 16 + r) * PL.lds + k0 + k]; }, g, t4);
#pragma unroll
      for (int j = 0; j < NZ; ++j) {
        const int n0 = (j * 8 + warp) * 8;
        if (n0 < Dp) {
          const T* b = sup + (n0 + g) * PL.ldu + k0 + t4;
          const uint32_t fb[2] = {__float_as_uint(DT<T>::to_f(b[0])), __float_as_uint(DT<T>::to_f(b[4]))};
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            mma_tf32(z[j][m], fa[m].lo, fb);
            mma_tf32(z[j][m], fa[m].hi, fb);
          }
        }
      }
    }
  }
  // ---- logarithms of the decays
#pragma unroll
  for (int j = 0; j < NZ; ++j) {
    const int n0 = (j * 8 + warp) * 8;
    if (n0 < Dp) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int d = n0 + 2 * t4 + i;
        const float b = d < D ? a.bias[rc + d] : 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int t = g + 8 * q;
          sp[t * ld + d] = t < n && d < D ? -a.c * sigmoidf(z[j][q >> 1][(q & 1) * 2 + i] + b) : 0.f;
        }
      }
    }
  }
  if (vec) {
#pragma unroll
    for (int u = 0; u < kEarly; ++u) file(tid + u * kThreads, early[u]);
    for (int i = tid + kEarly * kThreads; i < kC * per; i += kThreads) file(i, fetch(i));
  } else {
    for (int i = tid; i < kC * Dp; i += kThreads) {
      const int t = i / Dp, d = i % Dp;
      const bool on = t < n && d < D;
      const T* row = proj + (int64_t)t * a.ldp + d;
      sq[t * ld + d] = on ? DT<T>::to_f(row[rc]) : 0.f;
      sk[t * ld + d] = on ? DT<T>::to_f(row[kcol]) : 0.f;
      sb[t * ld + d] = on ? sigmoidf(DT<T>::to_f(row[acol]) + a.rate_bias[rc + d]) : 0.f;
    }
    for (int i = tid; i < kC * Vp; i += kThreads) {
      const int t = i / Vp, c = i % Vp;
      sv[t * ldv + c] = t < n && c < V ? proj[(int64_t)t * a.ldp + vcol + c] : DT<T>::from_f(0.f);
    }
  }
  __syncthreads();
  // ---- ... summed over the eight tokens of an item; lengths of the keys
  for (int i = tid; i < Dp * (kC / 8); i += kThreads) {
    const int d = i % Dp, b8 = i / Dp;
    float run = 0.f;
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      run += sp[(b8 * 8 + t) * ld + d];
      sp[(b8 * 8 + t) * ld + d] = run;
    }
    tot[b8 * (Dp + 1) + d] = run;
  }
  for (int t = warp; t < kC; t += kThreads / 32) {
    float kk = 0.f;
    for (int d = lane; d < Dp; d += 32) kk = fmaf(sk[t * ld + d], sk[t * ld + d], kk);
    kk = warp_sum(kk);
    if (lane == 0) sik[t] = 1.0f / sqrtf(kk + kUnitEps);
  }
  __syncthreads();
  // ---- p, q, b and g of the item's tokens; b of the whole chunk goes out
  for (int i = tid; i < Dp * (kC / 8); i += kThreads) {
    const int d = i % Dp, b8 = i / Dp, tb = b8 * 8;
    float before = 0.f, all = 0.f;
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float x = tot[q * (Dp + 1) + d];
      if (q < b8) before += x;
      all += x;
    }
    const float end = expf(all);
    float prev = expf(before);
    if (b8 == 0) out[L.g() + d] = d < D ? end : 0.f;
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const int at = (tb + t) * ld + d;
      const float l = before + sp[at], now = expf(l), inv = expf(-l);
      const float k = sk[at], u = k * sik[tb + t], bt = sb[at] * u * inv;
      sp[at] = prev * u;
      sq[at] = sq[at] * now;
      sk[at] = k * inv;
      sb[at] = bt;
      out[L.b() + (tb + t) * L.ldk + d] = bt * end;
      prev = now;
    }
  }
  if (L.Dm > Dp)
    for (int d = Dp + tid; d < L.Dm; d += kThreads) out[L.g() + d] = 0.f;
  __syncthreads();
  // ---- A, M (below the diagonal), H, E (with it): row tiles of [P; Q] (warp / 2), column tiles of [b; g]
  {
    const int m = warp >> 1, m0 = (m & 1) * 16, n0 = (warp & 1) * 32;
    const float* left = m < 2 ? sp : sq;
    const float* right = n0 == 0 ? sb : sk;
    const int nt = m0 == 0 ? 2 : 4;                       // column tiles that reach below the diagonal
    Acc acc[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j].zero();
    for (int k0 = 0; k0 < Dp; k0 += 8) {
      const FragA fa = frag_a([&](int r, int k) { return left[(m0 + r) * ld + k0 + k]; }, g, t4);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j < nt) acc[j].mac(fa, frag_b([&](int k, int c) { return right[(j * 8 + c) * ld + k0 + k]; }, g, t4));
    }
    float* dst = m < 2 ? (n0 == 0 ? mA : mM) : (n0 == 0 ? mH : mE);
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = m0 + g + 8 * (i >> 1), c = j * 8 + 2 * t4 + (i & 1);
        dst[t * kLdM + c] = (m < 2 ? c < t : c <= t) ? acc[j].get(i) : 0.f;
      }
  }
  __syncthreads();
  // ---- T = (I + A)^-1 by halves: two warps solve the 16 x 16 blocks on the diagonal, a lane per column ...
  if (warp < 2) {
    const int b = warp * 16;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float r0 = t == lane ? 1.f : 0.f, r1 = 0.f, r2 = 0.f, r3 = 0.f;
#pragma unroll
      for (int i = 0; i < t; i += 4) {
        const float4 w = *reinterpret_cast<const float4*>(mA + (b + t) * kLdM + b + i);
        r0 = fmaf(-w.x, x[i], r0);
        if (i + 1 < t) r1 = fmaf(-w.y, x[i + 1], r1);
        if (i + 2 < t) r2 = fmaf(-w.z, x[i + 2], r2);
        if (i + 3 < t) r3 = fmaf(-w.w, x[i + 3], r3);
      }
      x[t] = (r0 + r1) + (r2 + r3);
      if (lane < 16) mT[(b + t) * kLdM + b + lane] = x[t];
    }
  } else if (warp == 2) {
    for (int i = lane; i < 256; i += 32) mT[(i >> 4) * kLdM + 16 + (i & 15)] = 0.f;
  }
  __syncthreads();
  // ... and the block below is -T22 (A21 T11), eight columns per warp (A11's place holds the product in between)
  if (warp < 2) {
    const int n0 = warp * 8;
    Acc acc;
    acc.zero();
#pragma unroll
    for (int k0 = 0; k0 < 16; k0 += 8)
      acc.mac(frag_a([&](int r, int k) { return mA[(16 + r) * kLdM + k0 + k]; }, g, t4),
              frag_b([&](int k, int j) { return mT[(k0 + k) * kLdM + n0 + j]; }, g, t4));
#pragma unroll
    for (int i = 0; i < 4; ++i) mA[(g + 8 * (i >> 1)) * kLdM + n0 + 2 * t4 + (i & 1)] = acc.get(i);
    __syncwarp();
    acc.zero();
#pragma unroll
    for (int k0 = 0; k0 < 16; k0 += 8)
      acc.mac(frag_a([&](int r, int k) { return mT[(16 + r) * kLdM + 16 + k0 + k]; }, g, t4),
              frag_b([&](int k, int j) { return mA[(k0 + k) * kLdM + n0 + j]; }, g, t4));
#pragma unroll
    for (int i = 0; i < 4; ++i) mT[(16 + g + 8 * (i >> 1)) * kLdM + n0 + 2 * t4 + (i & 1)] = -acc.get(i);
  }
  __syncthreads();
  // ---- T M and H T: a warp has one 16 x 8 tile of each
  {
    const int m0 = (warp >> 2) * 16, n0 = (warp & 3) * 8;
    Acc x, y;
    x.zero();
    y.zero();
#pragma unroll
    for (int k0 = 0; k0 < kC; k0 += 8) {
      x.mac(frag_a([&](int r, int k) { return mT[(m0 + r) * kLdM + k0 + k]; }, g, t4),
            frag_b([&](int k, int j) { return mM[(k0 + k) * kLdM + n0 + j]; }, g, t4));
      y.mac(frag_a([&](int r, int k) { return mH[(m0 + r) * kLdM + k0 + k]; }, g, t4),
            frag_b([&](int k, int j) { return mT[(k0 + k) * kLdM + n0 + j]; }, g, t4));
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int at = (m0 + g + 8 * (i >> 1)) * kLdM + n0 + 2 * t4 + (i & 1);
      mTM[at] = x.get(i);
      mHT[at] = y.get(i);
    }
  }
  __syncthreads();
  // ---- E - H T M over E; W = T P and Q' = Q - H T P by 8-wide column tiles; g L_end - (T M)^T B over g
  {
    const int m0 = (warp >> 2) * 16, n0 = (warp & 3) * 8;
    Acc x;
    x.zero();
#pragma unroll
    for (int k0 = 0; k0 < kC; k0 += 8)
      x.mac(frag_a([&](int r, int k) { return mHT[(m0 + r) * kLdM + k0 + k]; }, g, t4),
            frag_b([&](int k, int j) { return mM[(k0 + k) * kLdM + n0 + j]; }, g, t4));
#pragma unroll
    for (int i = 0; i < 4; ++i) mE[(m0 + g + 8 * (i >> 1)) * kLdM + n0 + 2 * t4 + (i & 1)] -= x.get(i);
  }
  {
    // a warp keeps its row tile of [T; H T; (T M)^T] and walks the columns
    for (int m = 0; m < 6; ++m) {
      const int kind = m >> 1, m0 = (m & 1) * 16;
      const float* mat = kind == 0 ? mT : kind == 1 ? mHT : mTM;
      const int rs = kind == 2 ? 1 : kLdM, cs = kind == 2 ? kLdM : 1;
      FragA fm[4];
#pragma unroll
      for (int f = 0; f < 4; ++f)
        fm[f] = frag_a([&](int r, int k) { return mat[(m0 + r) * rs + (f * 8 + k) * cs]; }, g, t4);
      for (int n0 = warp * 8; n0 < Dp; n0 += kThreads / 4) {
        Acc x;
        x.zero();
        const float* src = kind == 2 ? sb : sp;
#pragma unroll
        for (int f = 0; f < 4; ++f)
          if (kind == 2 ? f * 8 + 8 > m0 : f * 8 <= m0 + 15)       // the matrices are triangular
            x.mac(fm[f], frag_b([&](int k, int j) { return src[(f * 8 + k) * ld + n0 + j]; }, g, t4));
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
          const int t = m0 + g + 4 * i, c = n0 + 2 * t4;
          if (kind == 0) {
            *reinterpret_cast<float2*>(out + t * L.ldw + c) = make_float2(x.get(i), x.get(i + 1));
          } else if (kind == 1) {
            *reinterpret_cast<float2*>(out + L.q() + t * L.ldw + c) =
                make_float2(sq[t * ld + c] - x.get(i), sq[t * ld + c + 1] - x.get(i + 1));
          } else {
            sk[t * ld + c] -= x.get(i);                // (times L_end below)
            sk[t * ld + c + 1] -= x.get(i + 1);
          }
        }
      }
    }
  }
  __syncthreads();
  // ---- Ob = (E - H T M) V and U = L_end (g - (T M)^T b)^T V by tiles of 16 rows; V is exact in one part
  const int rt = 2 + L.Dm / 16, ntile = Vp / 8;
  for (int tile = warp; tile < rt * (ntile / 4); tile += kThreads / 32) {
    const int m = tile / (ntile / 4), ng = tile % (ntile / 4);       // 32 columns: a slice
    float acc[4][4], low[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] = low[j][i] = 0.f;
    const int d0 = (m - 2) * 16;
    float e0 = 1.f, e1 = 1.f;
    if (m >= 2) {
      e0 = e1 = 0.f;
      float l0 = 0.f, l1 = 0.f;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (d0 + g < Dp) l0 += tot[q * (Dp + 1) + d0 + g];
        if (d0 + g + 8 < Dp) l1 += tot[q * (Dp + 1) + d0 + g + 8];
      }
      e0 = expf(l0);
      e1 = expf(l1);
    }
#pragma unroll
    for (int f = 0; f < 4; ++f) {
      const FragA fa = frag_a([&](int r, int k) {
        if (m < 2) return mE[(m * 16 + r) * kLdM + f * 8 + k];
        return d0 + r < Dp ? sk[(f * 8 + k) * ld + d0 + r] : 0.f;
      }, g, t4);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const T* v = sv + (f * 8 + t4) * ldv + ng * 32 + j * 8 + g;
        const uint32_t fb[2] = {__float_as_uint(DT<T>::to_f(v[0])), __float_as_uint(DT<T>::to_f(v[4 * ldv]))};
        mma_tf32(acc[j], fa.hi, fb);
        mma_tf32(low[j], fa.lo, fb);
      }
    }
    float* dst = out + L.slice(ng) + (m < 2 ? m * 16 : kC + d0) * L.ldu;
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        const float f = i == 0 ? e0 : e1;
        *reinterpret_cast<float2*>(dst + (g + 4 * i) * L.ldu + j * 8 + 2 * t4) =
            make_float2(f * (acc[j][i] + low[j][i]), f * (acc[j][i + 1] + low[j][i + 1]));
      }
  }
}

// CTA = 32 state columns of one head of one sequence; the state in accumulator fragments of MT row tiles per warp and a
// copy of it in shared memory, which the next chunk's products read.
template <int MT>
__global__ void __launch_bounds__(kThreads, 1) general_chunks_kernel(ChunkArgs s, int stages) {
  constexpr int N = 2;                                   // column tiles per warp
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(8) uint64_t full[4];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  const Common& a = s.c;
  const int D = a.dim, V = a.vdim, h = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * kVS, nv = min(kVS, V - v0);
  const Scratch L(D, V);
  const int Dp = L.Dp, Dm = L.Dm, ldw = L.ldw, ldk = L.ldk, ldu = L.ldu;
  const int first = s.seq_chunk[seq], last = s.seq_chunk[seq + 1];
  const int ca = max(first, s.c0), cb = min(last, s.c1);
  if (ca >= cb) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  float* stage0 = sm;
  float* sS = stage0 + stages * L.stage();               // [Dm][40]
  float* sX = sS + Dm * ldu;                             // [32][40]
  const int row0 = a.seq_row[seq], len = a.seq_len[seq];
  const int slot = a.slot[row0], start = a.start[slot], p0 = a.pos[row0];
  float* st = a.state + (((int64_t)slot * a.heads + h) * D) * V + v0;
  auto fetch = [&](int c) {                              // one thread
    if (c >= cb) return;
    const float* src = s.scratch + ((int64_t)(c - s.c0) * a.heads + h) * L.floats();
    float* dst = stage0 + ((c - ca) % stages) * L.stage();
    uint64_t* bar = &full[(c - ca) % stages];
    tc5::mbar_expect_tx(bar, (uint32_t)(L.stage() * sizeof(float)));
    bulk_load(dst, src, (uint32_t)(L.shared_part() * sizeof(float)), bar);
    bulk_load(dst + L.shared_part(), src + L.slice(blockIdx.x), (uint32_t)(L.slice_part() * sizeof(float)), bar);
  };
  if (tid == 0) {
    for (int i = 0; i < 4; ++i) tc5::mbar_init(&full[i], 1);
    abort_word = 0;
    tc5::fence_barrier_init();
    for (int i = 0; i < stages; ++i) fetch(ca + i);
  }
  const int wm = warp >> 1, wn = (warp & 1) * N;         // row tiles wm, wm + 4, ..., column tiles wn, wn + 1
  float S[MT][N][4];
  const bool fresh = ca == first && p0 <= start;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (wm + 4 * m) * 16 + g + 8 * (i >> 1), c = (wn + n) * 8 + 2 * t4 + (i & 1);
        S[m][n][i] = !fresh && d < D && c < nv ? st[(int64_t)d * V + c] : 0.f;
        if (d < Dm) sS[d * ldu + c] = S[m][n][i];
      }
  const int mt = warp >> 1;                              // row tile of [W; Q'], 0 .. 3
  bool ok = true;
  for (int c = ca; c < cb; ++c) {
    __syncthreads();                                     // the state is in place (and, first, the barriers)
    if (!tc5::mbar_wait(&full[(c - ca) % stages], ((c - ca) / stages) & 1, abort_flag)) {
      if (lane == 0) tc5::report(s.err, 42);
      ok = false;
      break;
    }
    const float* b0 = stage0 + ((c - ca) % stages) * L.stage();
    const float *B = b0 + L.b(), *G = b0 + L.g(), *Ob = b0 + L.shared_part(), *U = Ob + kC * ldu;
    Acc acc[N];
#pragma unroll
    for (int n = 0; n < N; ++n) acc[n].zero();
    {
      const float* left = b0 + mt * 16 * ldw;            // Q' follows W
#pragma unroll 4
      for (int k0 = 0; k0 < Dp; k0 += 8) {
        const FragA fa = frag_a([&](int r, int k) { return left[r * ldw + k0 + k]; }, g, t4);
#pragma unroll
        for (int n = 0; n < N; ++n)
          acc[n].mac(fa, frag_b([&](int k, int j) { return sS[(k0 + k) * ldu + (wn + n) * 8 + j]; }, g, t4));
      }
    }
    if (mt < 2) {
#pragma unroll
      for (int n = 0; n < N; ++n)
#pragma unroll
        for (int i = 0; i < 4; i += 2)
          *reinterpret_cast<float2*>(sX + (mt * 16 + g + 4 * i) * ldu + (wn + n) * 8 + 2 * t4) =
              make_float2(acc[n].get(i), acc[n].get(i + 1));
    }
    __syncthreads();                                     // X is complete, the old state is read
    if (mt >= 2) {
      const int off = (c - first) * kC;
#pragma unroll
      for (int n = 0; n < N; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int t = (mt - 2) * 16 + g + 8 * (i >> 1), col = (wn + n) * 8 + 2 * t4 + (i & 1);
          if (off + t < len && col < nv)
            s.raw[((int64_t)(row0 + off + t) * a.heads + h) * V + v0 + col] = Ob[t * ldu + col] + acc[n].get(i);
        }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int d0 = (wm + 4 * m) * 16;
      if (d0 < Dm) {
        Acc down[N];
#pragma unroll
        for (int n = 0; n < N; ++n) down[n].zero();
#pragma unroll
        for (int k0 = 0; k0 < kC; k0 += 8) {
          const FragA fa = frag_a([&](int r, int k) { return d0 + r < Dp ? B[(k0 + k) * ldk + d0 + r] : 0.f; }, g, t4);
#pragma unroll
          for (int n = 0; n < N; ++n)
            down[n].mac(fa, frag_b([&](int k, int j) { return sX[(k0 + k) * ldu + (wn + n) * 8 + j]; }, g, t4));
        }
        const float g0 = G[d0 + g], g1 = G[d0 + g + 8];
#pragma unroll
        for (int n = 0; n < N; ++n)
#pragma unroll
          for (int i = 0; i < 4; i += 2) {
            const int at = (d0 + g + 4 * i) * ldu + (wn + n) * 8 + 2 * t4;
            const float2 u = *reinterpret_cast<const float2*>(U + at);
            const float f = i == 0 ? g0 : g1;
            S[m][n][i] = fmaf(f, S[m][n][i], u.x - down[n].get(i));
            S[m][n][i + 1] = fmaf(f, S[m][n][i + 1], u.y - down[n].get(i + 1));
            *reinterpret_cast<float2*>(sS + at) = make_float2(S[m][n][i], S[m][n][i + 1]);
          }
      }
    }
    __syncthreads();                                     // the stage and X are free again
    if (tid == 0) fetch(c + stages);
  }
  if (!ok) {                                             // copies in flight still write to this CTA's memory
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
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (wm + 4 * m) * 16 + g + 8 * (i >> 1), c = (wn + n) * 8 + 2 * t4 + (i & 1);
        if (d < D && c < nv) st[(int64_t)d * V + c] = S[m][n][i];
      }
}

bool sizes_ok(int heads, int dim, int vdim, int rank) {
  return heads >= 1 && heads <= 65535 && dim >= 1 && dim <= 512 && vdim >= 1 && vdim <= 65535 && rank >= 1;
}

template <typename T, int NR, int CV>
cudaError_t launch_step(StepArgs& s, int seqs, bool fused, bool pdl, cudaStream_t st) {
  const int slices = (s.c.vdim + 32 * CV - 1) / (32 * CV);
  if (fused && slices > 8) return cudaErrorInvalidValue;
  size_t smem = (2 * (4 * (size_t)s.c.dim + 32 * CV) + 2 * 2 * 8 * 32 * CV + 2 * (size_t)s.c.rank) * sizeof(float);
  const size_t up = (size_t)s.c.dim * (s.c.rank | 1) * sizeof(float);
  s.staged = smem + up <= 100 * 1024;
  if (s.staged) smem += up;
  if (smem > kSmemMax) return cudaErrorInvalidValue;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(general_step_kernel<T, NR, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
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
  return cudaLaunchKernelEx(&cfg, general_step_kernel<T, NR, CV>, s);
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

Common common_args(const void* proj, int64_t ldp, const float* low, int64_t ldl, const void* up, const float* bias,
                   const float* rate_bias, float* state, const int* slot, const int* pos, const int* start,
                   const int* seq_row, const int* seq_len, int heads, int dim, int vdim, int rank, float c) {
  return Common{proj, low, up, bias, rate_bias, state, slot, pos, start, seq_row, seq_len, ldp, ldl, heads, dim, vdim, rank, c};
}

}  // namespace

// Can the chunked form take these sizes and decays of at least exp(-c)?
IPEX_API int ipex_general_chunks_ok(int dim, int vdim, int rank, float c) {
  const Scratch L(dim, vdim);
  return dim >= 1 && dim <= 256 && vdim >= 1 && rank >= 1 && c >= 0.f && c * kC <= kMaxLog && prep_smem(L) <= kSmemMax &&
         chunk_smem(L, 1) <= kSmemMax;
}
IPEX_API int64_t ipex_general_scratch_floats(int dim, int vdim) { return Scratch(dim, vdim).floats(); }
// Can a decode step of these sizes norm its outputs on the way?
IPEX_API int ipex_general_fused_ok(int vdim) { return vdim >= 1 && vdim <= 256; }

// Token by token.  seq_row / seq_len null: `seqs` sequences of one token each; norm_w [heads * vdim] / out [tokens, ldo] then
// take norm(o) * norm_w * sigmoid(gate) (vdim <= 256; out may be the gates' place).  raw (when out is null): the plain
// outputs [tokens, heads, vdim].
IPEX_API int ipex_general_step(const void* proj, int64_t ldp, int gate_off, const float* low, int64_t ldl, const void* up,
                               const float* bias, const float* rate_bias, float* state, const int* slot, const int* pos,
                               const int* start, const int* seq_row, const int* seq_len, int seqs, const void* norm_w,
                               float eps, void* out, int64_t ldo, float* raw, int heads, int dim, int vdim, int rank, float c,
                               int dtype, int pdl, void* stream) {
  if (!sizes_ok(heads, dim, vdim, rank) || seqs < 1 || seqs > 65535 || (seq_row == nullptr) != (seq_len == nullptr))
    return (int)cudaErrorInvalidValue;
  const bool fused = raw == nullptr;
  if (fused && (seq_row != nullptr || out == nullptr || norm_w == nullptr || !ipex_general_fused_ok(vdim)))
    return (int)cudaErrorInvalidValue;
  return by_dtype(dtype, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    StepArgs s = {common_args(proj, ldp, low, ldl, up, bias, rate_bias, state, slot, pos, start, seq_row, seq_len, heads, dim,
                              vdim, rank, c),
                  norm_w, out, raw, ldo, eps, gate_off, pdl && fused && vdim % 4 == 0, 0};
    cudaStream_t st = (cudaStream_t)stream;
    if (dim <= 32) return pick_cols<T, 4>(s, seqs, fused, pdl != 0, st);
    if (dim <= 64) return pick_cols<T, 8>(s, seqs, fused, pdl != 0, st);
    if (dim <= 128) return pick_cols<T, 16>(s, seqs, fused, pdl != 0, st);
    if (dim <= 256) return pick_cols<T, 32>(s, seqs, fused, pdl != 0, st);
    return pick_cols<T, 64>(s, seqs, fused, pdl != 0, st);
  });
}

// Chunks [c0, c1) of a packed batch in the chunked form (16-bit models).  chunk_seq [chunks], seq_chunk [seqs + 1]: device
// tables of the sequences' chunks of 32 tokens, in order; scratch: (c1 - c0) * heads * ipex_general_scratch_floats; raw as
// above.
IPEX_API int ipex_general_chunks(const void* proj, int64_t ldp, const float* low, int64_t ldl, const void* up,
                                 const float* bias, const float* rate_bias, float* state, const int* slot, const int* pos,
                                 const int* start, const int* seq_row, const int* seq_len, int seqs, const int* chunk_seq,
                                 const int* seq_chunk, int c0, int c1, float* scratch, float* raw, int heads, int dim,
                                 int vdim, int rank, float c, int dtype, int* err, void* stream) {
  if (!sizes_ok(heads, dim, vdim, rank) || !ipex_general_chunks_ok(dim, vdim, rank, c) || seqs < 1 || seqs > 65535 ||
      c0 < 0 || c1 <= c0 || seq_row == nullptr || seq_len == nullptr || (((uintptr_t)scratch) & 15) || dtype == DT_F32)
    return (int)cudaErrorInvalidValue;
  auto run = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ChunkArgs s = {common_args(proj, ldp, low, ldl, up, bias, rate_bias, state, slot, pos, start, seq_row, seq_len, heads, dim,
                               vdim, rank, c),
                   chunk_seq, seq_chunk, scratch, raw, err, c0, c1};
    cudaStream_t st = (cudaStream_t)stream;
    const Scratch L(dim, vdim);
    const size_t ps = prep_smem(L);
    auto prep = dim <= 64 ? general_prep_kernel<T, 1> : dim <= 128 ? general_prep_kernel<T, 2> : general_prep_kernel<T, 4>;
    cudaError_t e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ps);
    if (e != cudaSuccess) return e;
    prep<<<dim3(c1 - c0, heads), kThreads, ps, st>>>(s);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    int stages = 3;
    while (stages > 1 && chunk_smem(L, stages) > kSmemMax) --stages;
    const size_t cs = chunk_smem(L, stages);
    auto kern = dim <= 64 ? general_chunks_kernel<1> : dim <= 128 ? general_chunks_kernel<2> : general_chunks_kernel<4>;
    e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cs);
    if (e != cudaSuccess) return e;
    kern<<<dim3(L.slices, heads, seqs), kThreads, cs, st>>>(s, stages);
    return cudaGetLastError();
  };
  return (int)(dtype == DT_F16 ? run((__half*)nullptr) : run((__nv_bfloat16*)nullptr));
}
