// Prompt attention over packed sequences on the 5th-generation tensor cores, sm_100a: multi-head latent attention, and
// attention with plain key / value heads (shared by groups of query heads), over everything earlier, a window (alone or
// beside pooled blocks of the tokens before it) or the query's own chunk, with or without a sink and an output gate.
//
// Keys and values are expanded from the latents by two GEMMs before this kernel; a head's key is then made of two
// parts that live in different tensors: `dim` values of its own and `rd` rotated values shared by all heads.  Neither
// part is copied together: the score is accumulated over 64-wide k-blocks, and every block comes straight from its
// own tensor through TMA (zero-filled past `dim` or `rd`):
//
//   S  = sum over blocks of  Q_blk [128 x 64] . K_blk [128 x 64]^T   -> TMEM columns [0, 128) and [128, 256), alternating
//   PV = P [128 queries x 128 keys] . V^T tile [DV x 128 keys]       -> TMEM columns [256, 256 + DV)
//
// V^T is produced directly by a GEMM with W_uv as its row operand.  Sequences of different lengths are packed one
// behind the other (no padding rows); a CTA owns 128 queries of one head of one sequence and walks the key tiles
// inside the causal sliding window.  A V^T tile must start at a multiple of 8 tokens (16-byte TMA rule), so tiles are
// laid out from the sequence's first row rounded down to 8 and the surplus keys are masked.  Pooled blocks are keys and
// values of their own tensors, in rows that start at multiples of 8; their tiles come first.
//
//   warp 8: TMA loads (separate rings for K and V^T)   warp 9: MMA issue, S(j+1) goes out before P(j) is waited for
//   warps 0-7: two threads per query row: maximum, exp2, sum, P to shared memory, running output in registers
//
// Every mbarrier wait is bounded; a wait that runs out raises the CTA's abort flag, the error word gets a code
// (34 loader, 35 MMA issuer, 36 softmax) and all roles leave, after which TMEM is freed.
#include "common/utils.cuh"
#include "tcgen05_common.cuh"

namespace {

using namespace tc5;

constexpr int kBQ = 128, kBKV = 128;
constexpr int kThreads = 320;
constexpr int kBlkBytes = 128 * 128;      // one 128-row x 64-element operand block

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* tm, int x, int y, int z, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(tm)), "r"(x), "r"(y), "r"(z), "r"(smem_u32(bar))
      : "memory");
}

struct Args {
  void* out;              // T [tokens, ldo], head h at h * vd
  const int* seq_row;     // [B] first packed row of every sequence
  const int* seq_len;     // [B]
  int* err;
  int64_t ldo;
  int dim, rd, vd, window;
  int nbn, nbr;           // k-blocks of the own and of the shared part
  int kst, vst;           // stages of the K and V^T rings (1 or 2)
  int group;              // query heads per key / value head
  int sink;               // one more score, without a value, in every softmax: 0, or sinks[head]
  float scale_log2;
  int chunk;              // keys of the query's own chunk of this many positions only; 0: all
  const float* sinks;
  const void* gate;       // T [tokens, ldg], head h at h * vd, or null: outputs times gate_scale * sigmoid(gate)
  int64_t ldg;
  float gate_scale;
  int pool;               // > 0: beside the window, the blocks of this many tokens that lie wholly before it
  const int* pool_row;    // [B] first row of every sequence's blocks, a multiple of 8
};

template <typename T, int DV>
__global__ void __launch_bounds__(kThreads, 1)
packed_prefill_kernel(const __grid_constant__ CUtensorMap tm_qn, const __grid_constant__ CUtensorMap tm_qr,
                      const __grid_constant__ CUtensorMap tm_kn, const __grid_constant__ CUtensorMap tm_kr,
                      const __grid_constant__ CUtensorMap tm_vt, const __grid_constant__ CUtensorMap tm_kp,
                      const __grid_constant__ CUtensorMap tm_vp, Args a) {
  constexpr int kVBytes = DV * kBKV * 2;
  constexpr uint32_t kTmemCols = 512;
  const int h = blockIdx.x, b = blockIdx.z, hk = h / a.group;
  const int len = a.seq_len[b], row0 = a.seq_row[b];
  const int nqb = (len + kBQ - 1) / kBQ;
  const int qb = (int)gridDim.y - 1 - (int)blockIdx.y;      // longest rows of the longest sequence first
  if (qb >= nqb) return;
  const int nb = a.nbn + a.nbr;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sP = sQ + nb * kBlkBytes;
  uint8_t* sK = sP + 2 * kBlkBytes;
  uint8_t* sV = sK + a.kst * nb * kBlkBytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + a.vst * kVBytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;      // [2]
  uint64_t* p_full = bars + 11;
  uint64_t* o_full = bars + 12;
  uint64_t* o_free = bars + 13;
  uint64_t* x_full = bars + 14;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* xch = reinterpret_cast<float*>(bars + 32);          // [2][128]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int koff = row0 & 7, base = row0 - koff;             // tile j, column i <-> key j * 128 + i - koff
  const int qmax = min(qb * kBQ + kBQ, len) - 1;
  const int nkv = (qmax + koff) / kBKV + 1;
  int j0 = 0;
  if (a.window > 0) j0 = max(0, qb * kBQ - a.window + 1 + koff) / kBKV;
  if (a.chunk > 0) j0 = max(j0, (qb * kBQ / a.chunk * a.chunk + koff) / kBKV);
  // tiles of pooled blocks that some row sees, then those of tokens
  const int npt = a.pool > 0 ? (max(0, qmax - a.window + 1) / a.pool + kBKV - 1) / kBKV : 0;
  const int prow = a.pool > 0 ? a.pool_row[b] : 0;
  const int nblk = npt + nkv - j0;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1);
    }
    mbar_init(p_full, 256);
    mbar_init(o_full, 1);
    mbar_init(o_free, 256);
    mbar_init(x_full, 256);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 9) tmem_alloc(tmem_slot, kTmemCols);
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 8) {
    // ---------------- loader ----------------
    if (lane == 0) {
      mbar_expect_tx(q_full, nb * kBlkBytes);
      for (int i = 0; i < a.nbn; ++i) tma_load_3d(sQ + i * kBlkBytes, &tm_qn, i * 64, h, row0 + qb * kBQ, q_full);
      for (int i = 0; i < a.nbr; ++i)
        tma_load_3d(sQ + (a.nbn + i) * kBlkBytes, &tm_qr, i * 64, h, row0 + qb * kBQ, q_full);
      bool ok = true;
      int ks = 0, vs = 0;
      uint32_t kp = 0, vp = 0;
      for (int jj = 0; jj < nblk && ok; ++jj) {
        const bool pooled = jj < npt;
        const CUtensorMap* tk = pooled ? &tm_kp : &tm_kn;
        const CUtensorMap* tv = pooled ? &tm_vp : &tm_vt;
        const int krow = pooled ? prow + jj * kBKV : base + (j0 + jj - npt) * kBKV;
        if (!mbar_wait(&k_empty[ks], kp ^ 1, abort_flag)) { ok = false; report(a.err, 34); break; }
        uint8_t* dk = sK + ks * nb * kBlkBytes;
        mbar_expect_tx(&k_full[ks], nb * kBlkBytes);
        for (int i = 0; i < a.nbn; ++i) tma_load_3d(dk + i * kBlkBytes, tk, i * 64, hk, krow, &k_full[ks]);
        for (int i = 0; i < a.nbr; ++i) tma_load_2d(dk + (a.nbn + i) * kBlkBytes, &tm_kr, i * 64, krow, &k_full[ks]);
        if (++ks == a.kst) { ks = 0; kp ^= 1; }
        if (!mbar_wait(&v_empty[vs], vp ^ 1, abort_flag)) { ok = false; report(a.err, 34); break; }
        uint8_t* dv = sV + vs * kVBytes;
        mbar_expect_tx(&v_full[vs], kVBytes);
#pragma unroll
        for (int i = 0; i < kBKV / 64; ++i)
          tma_load_2d(dv + i * (DV * 128), tv, krow + i * 64, hk * a.vd, &v_full[vs]);
        if (++vs == a.vst) { vs = 0; vp ^= 1; }
      }
      if (!ok) {
        mbar_wait_quiet(q_full, 0, 1 << 12);
        for (int i = 0; i < 2; ++i) {
          mbar_wait_quiet(&k_full[i], 0, 1 << 12);
          mbar_wait_quiet(&v_full[i], 0, 1 << 12);
        }
      }
    }
    __syncwarp();
  } else if (warp == 9) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_f16<T>(kBQ, kBKV);
      const uint32_t idesc_o = make_idesc_f16<T>(kBQ, DV);
      const uint32_t tm_o = tmem_base + 2 * kBKV;
      int ks = 0, vs = 0;
      uint32_t kp = 0, vp = 0;
      auto scores = [&](int jj) {       // S(jj) into score buffer jj & 1
        if (!mbar_wait(&k_full[ks], kp, abort_flag)) return false;
        tcgen05_fence_after();
        const uint32_t tm_s = tmem_base + (jj & 1) * kBKV;
        const uint8_t* kb = sK + ks * nb * kBlkBytes;
        for (int i = 0; i < nb; ++i) {
          const uint64_t ad = make_desc_sw128(smem_u32(sQ + i * kBlkBytes));
          const uint64_t bd = make_desc_sw128(smem_u32(kb + i * kBlkBytes));
          const int width = i < a.nbn ? a.dim - i * 64 : a.rd - (i - a.nbn) * 64;
          const int steps = width >= 64 ? 4 : (width + 15) / 16;
          for (int kk = 0; kk < steps; ++kk) umma_f16(tm_s, ad + 2 * kk, bd + 2 * kk, idesc_s, (i | kk) != 0);
        }
        umma_commit(&s_full[jj & 1]);
        umma_commit(&k_empty[ks]);
        if (++ks == a.kst) { ks = 0; kp ^= 1; }
        return true;
      };
      bool ok = mbar_wait(q_full, 0, abort_flag) && scores(0);
      for (int jj = 0; jj < nblk && ok; ++jj) {
        const uint32_t jp = jj & 1;
        // the other score buffer was read before p_full(jj - 1), which the previous iteration waited for
        if (jj + 1 < nblk && !scores(jj + 1)) { ok = false; break; }
        if (!mbar_wait(&v_full[vs], vp, abort_flag)) { ok = false; break; }
        if (!mbar_wait(p_full, jp, abort_flag)) { ok = false; break; }
        if (jj > 0 && !mbar_wait(o_free, jp ^ 1, abort_flag)) { ok = false; break; }
        tcgen05_fence_after();
        const uint8_t* vb = sV + vs * kVBytes;
#pragma unroll
        for (int i = 0; i < kBKV / 64; ++i) {
          const uint64_t ad = make_desc_sw128(smem_u32(sP + i * kBlkBytes));
          const uint64_t bd = make_desc_sw128(smem_u32(vb + i * (DV * 128)));
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_f16(tm_o, ad + 2 * kk, bd + 2 * kk, idesc_o, (i | kk) != 0);
        }
        umma_commit(o_full);
        umma_commit(&v_empty[vs]);
        if (++vs == a.vst) { vs = 0; vp ^= 1; }
      }
      if (!ok) report(a.err, 35);
    }
    __syncwarp();
  } else {
    // ---------------- softmax + output ----------------
    const int r = threadIdx.x & 127, hf = threadIdx.x >> 7;
    const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
    const int qpos = qb * kBQ + r;
    constexpr int kOH = DV / 2;
    float o[kOH];
#pragma unroll
    for (int d = 0; d < kOH; ++d) o[d] = 0.f;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    int first = a.window > 0 ? max(0, qpos - a.window + 1) : 0;
    if (a.chunk > 0) first = max(first, qpos / a.chunk * a.chunk);
    const int seen = a.pool > 0 ? max(0, qpos - a.window + 1) / a.pool : 0;      // blocks that this row sees
    for (int jj = 0; jj < nblk; ++jj) {
      const uint32_t jp = jj & 1;
      if (!mbar_wait(&s_full[jj & 1], (jj >> 1) & 1, abort_flag)) { ok = false; break; }
      tcgen05_fence_after();
      const bool pooled = jj < npt;
      // key of this thread's first column, visible columns [lo, lim)
      const int k0 = pooled ? jj * kBKV + hf * 64 : (j0 + jj - npt) * kBKV - koff + hf * 64;
      const int lim = (pooled ? seen : qpos + 1) - k0, lo = pooled ? 0 : first - k0;
      uint32_t v0[32], v1[32];
      const uint32_t sb = tmem_base + lane_addr + (jj & 1) * kBKV + hf * 64;
      tmem_ld_32x32(sb, v0);
      tmem_ld_32x32(sb + 32, v1);
      float mx = -INFINITY;
      const bool full = lim >= 64 && lo <= 0;
      if (full) {
#pragma unroll
        for (int i = 0; i < 32; ++i) mx = fmaxf(mx, fmaxf(__uint_as_float(v0[i]), __uint_as_float(v1[i])));
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          if (i < lim && i >= lo) mx = fmaxf(mx, __uint_as_float(v0[i]));
          if (32 + i < lim && 32 + i >= lo) mx = fmaxf(mx, __uint_as_float(v1[i]));
        }
      }
      if (a.scale_log2 >= 0.f) {
        mx = mx == -INFINITY ? mx : mx * a.scale_log2;
      } else if (mx != -INFINITY) {                          // a negative scale reverses the order of the scores
        mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          if (i < lim && i >= lo) mx = fmaxf(mx, __uint_as_float(v0[i]) * a.scale_log2);
          if (32 + i < lim && 32 + i >= lo) mx = fmaxf(mx, __uint_as_float(v1[i]) * a.scale_log2);
        }
      }
      xch[hf * 128 + r] = mx;
      mbar_arrive(x_full);
      if (!mbar_wait(x_full, jp, abort_flag)) { ok = false; break; }
      mx = fmaxf(fmaxf(mx, xch[(hf ^ 1) * 128 + r]), m);
      const float mref = mx == -INFINITY ? 0.f : mx;
      const float corr = ex2(m - mref);
      float psum = 0.f;
      uint8_t* prow = sP + hf * kBlkBytes + r * 128;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        __align__(16) T pk[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const float sv = __uint_as_float(half == 0 ? v0[i] : v1[i]);
          float p = ex2(fmaf(sv, a.scale_log2, -mref));
          if (!full && (half * 32 + i >= lim || half * 32 + i < lo)) p = 0.f;
          const T pt = from_float<T>(p);
          pk[i] = pt;
          psum += to_float<T>(pt);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int chunk = half * 4 + q;
          *reinterpret_cast<uint4*>(prow + ((chunk ^ (r & 7)) << 4)) = reinterpret_cast<const uint4*>(pk)[q];
        }
      }
      l = l * corr + psum;
      m = mx;
      fence_proxy_async_smem();
      tcgen05_fence_before();
      mbar_arrive(p_full);
      if (!mbar_wait(o_full, jp, abort_flag)) { ok = false; break; }
      tcgen05_fence_after();
#pragma unroll
      for (int c = 0; c < kOH / 32; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(tmem_base + lane_addr + 2 * kBKV + hf * kOH + c * 32, v);
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(o[c * 32 + i], corr, __uint_as_float(v[i]));
      }
      tcgen05_fence_before();
      mbar_arrive(o_free);
    }
    if (ok) {
      xch[hf * 128 + r] = l;
      mbar_arrive(x_full);
      ok = mbar_wait(x_full, nblk & 1, abort_flag);
      l += xch[(hf ^ 1) * 128 + r];
      if (a.sink) {                  // both halves hold the row's maximum, in the log2 domain
        const float z = a.sinks != nullptr ? a.sinks[h] * 1.4426950408889634f : 0.f;
        const float top = fmaxf(m, z), f = ex2(m - top);
        l = l * f + ex2(z - top);
#pragma unroll
        for (int d = 0; d < kOH; ++d) o[d] *= f;
      }
    }
    if (!ok && lane == 0) report(a.err, 36);
    if (ok && qpos < len) {
      const float inv = l > 0.f ? 1.f / l : 0.f;
      T* op = reinterpret_cast<T*>(a.out) + (int64_t)(row0 + qpos) * a.ldo + (int64_t)h * a.vd + hf * kOH;
      const T* gp = reinterpret_cast<const T*>(a.gate) + (int64_t)(row0 + qpos) * a.ldg + (int64_t)h * a.vd + hf * kOH;
#pragma unroll
      for (int c = 0; c < kOH / 8; ++c) {
        if (hf * kOH + c * 8 < a.vd) {
          __align__(16) T ov[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) o[c * 8 + i] *= inv;
          if (a.gate != nullptr) {
            const uint4 raw = *reinterpret_cast<const uint4*>(gp + c * 8);
            const T* gv = reinterpret_cast<const T*>(&raw);
#pragma unroll
            for (int i = 0; i < 8; ++i) o[c * 8 + i] *= __fdividef(a.gate_scale, 1.0f + __expf(-to_float<T>(gv[i])));
          }
#pragma unroll
          for (int i = 0; i < 8; ++i) ov[i] = from_float<T>(o[c * 8 + i]);
          *reinterpret_cast<uint4*>(op + c * 8) = *reinterpret_cast<const uint4*>(ov);
        }
      }
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 9) tmem_dealloc(tmem_base, kTmemCols);
}

// 3-D map (width, heads, rows) of a row-major activation: box 64 x 1 x 128 in the 128-byte swizzle, zeros outside.
bool encode_heads(CUtensorMap* tm, CUtensorMapDataType dt, const void* base, int width, int heads, int64_t rows,
                  int64_t head_stride, int64_t row_stride) {
  EncodeTiledFn enc = tensor_map_encoder();
  if (enc == nullptr) return false;
  cuuint64_t dims[3] = {(cuuint64_t)width, (cuuint64_t)heads, (cuuint64_t)rows};
  cuuint64_t strides[2] = {(cuuint64_t)head_stride * 2, (cuuint64_t)row_stride * 2};
  cuuint32_t box[3] = {64, 1, 128};
  cuuint32_t estr[3] = {1, 1, 1};
  return enc(tm, dt, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

constexpr size_t kSmemMax = 227 * 1024;
size_t smem_need(int nb, int dv, int kst, int vst) {
  return 1024 + (size_t)(nb + 2 + kst * nb) * kBlkBytes + (size_t)vst * dv * kBKV * 2 + 256 + 1024;
}

template <typename T, int DV>
int launch(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* kr, int64_t ld_kr, const void* vt,
           int64_t ld_vt, const void* kp, int64_t ld_kp, const void* vp, int64_t ld_vp, int pool_rows, Args& a, int B, int H,
           int tokens, int max_len, cudaStream_t stream) {
  const CUtensorMapDataType dt =
      std::is_same<T, __half>::value ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const int nb = a.nbn + a.nbr;
  a.kst = a.vst = 2;
  if (smem_need(nb, DV, 2, 2) > kSmemMax) a.vst = 1;
  if (smem_need(nb, DV, 2, a.vst) > kSmemMax) a.kst = 1;
  const size_t smem = smem_need(nb, DV, a.kst, a.vst);
  if (smem > kSmemMax) return (int)cudaErrorInvalidValue;
  CUtensorMap qn, qr, kn, krm, vm, kpm, vpm;
  const T* qp = reinterpret_cast<const T*>(q);
  const int G = H / a.group;
  if (!encode_heads(&qn, dt, qp, a.dim, H, tokens, a.dim + a.rd, ldq) ||
      !encode_heads(&kn, dt, k, a.dim, G, tokens, a.dim, ldk) ||
      !encode_2d_sw128(&vm, dt, vt, (uint64_t)tokens, (uint64_t)G * a.vd, (uint64_t)ld_vt * 2, 64, DV))
    return -1;
  qr = qn;
  krm = qn;
  if (a.nbr > 0 && (!encode_heads(&qr, dt, qp + a.dim, a.rd, H, tokens, a.dim + a.rd, ldq) ||
                    !encode_2d_sw128(&krm, dt, kr, (uint64_t)a.rd, (uint64_t)tokens, (uint64_t)ld_kr * 2, 64, kBKV)))
    return -1;
  kpm = kn;
  vpm = vm;
  if (a.pool > 0 && (!encode_heads(&kpm, dt, kp, a.dim, G, pool_rows, a.dim, ld_kp) ||
                     !encode_2d_sw128(&vpm, dt, vp, (uint64_t)pool_rows, (uint64_t)G * a.vd, (uint64_t)ld_vp * 2, 64, DV)))
    return -1;
  auto kern = packed_prefill_kernel<T, DV>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  dim3 grid(H, (max_len + kBQ - 1) / kBQ, B);
  kern<<<grid, kThreads, smem, stream>>>(qn, qr, kn, krm, vm, kpm, vpm, a);
  return (int)cudaGetLastError();
}

}  // namespace

// Sizes the kernel takes: parts that keep every TMA stride a multiple of 16 bytes, at most 256 score columns in
// 64-wide blocks, values up to 128.
IPEX_API int ipex_packed_prefill_ok(int dim, int rd, int vd, int R, int dtype) {
  if (dtype != DT_F16 && dtype != DT_BF16) return 0;
  if (dim < 8 || rd < 0 || vd < 8 || (dim % 8) || (rd % 8) || (vd % 8) || (R % 8)) return 0;
  return (dim + 63) / 64 + (rd + 63) / 64 <= 4 && vd <= 128;
}

// Causal (windowed) attention of packed sequences: q [tokens, ldq] holds per head [dim | rd (rotated)], k [tokens, ldk]
// the G key heads of `dim`, kr [tokens, ld_kr] the rotated part shared by all heads (rd = 0: none), vt [G * vd, ld_vt]
// the values transposed.  Query head h uses key / value head h / (H / G).  seq_row / seq_len: device, [B]; max_len: the
// largest length.  window 0: unlimited.  chunk > 0: keys of the query's own chunk only.  sink: every softmax has one more
// score, 0 or sinks[head], whose value is nothing.  pool > 0 (with a window, rd = 0): beside the window the blocks of `pool`
// tokens that lie wholly before it, keys kp [pool_rows, ld_kp] and transposed values vp [G * vd, ld_vp] in rows from
// pool_row[sequence] (device, multiples of 8) on; rows that are no block must hold finite numbers.  gate (may be null): [tokens, ldg], outputs times gate_scale *
// sigmoid(gate).  Strides multiples of 8 elements, bases 16-byte aligned.  Returns a cudaError_t, or -1 when the tensor-map encoder rejects
// the operands.
IPEX_API int ipex_packed_prefill(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* kr, int64_t ld_kr,
                                 const void* vt, int64_t ld_vt, void* out, int64_t ldo, const int* seq_row,
                                 const int* seq_len, int B, int H, int G, int tokens, int max_len, int dim, int rd,
                                 int vd, int window, int chunk, int sink, const float* sinks, const void* gate,
                                 int64_t ldg, float gate_scale, int pool, const void* kp, int64_t ld_kp, const void* vp,
                                 int64_t ld_vp, const int* pool_row, int pool_rows, float scale, int dtype, int* err,
                                 void* stream) {
  if (!ipex_packed_prefill_ok(dim, rd, vd, 8, dtype) || B < 1 || B > 65535 || H < 1 || tokens < 1 || max_len < 1 ||
      window < 0 || chunk < 0 || (max_len + kBQ - 1) / kBQ > 65535 || G < 1 || H % G != 0)
    return (int)cudaErrorInvalidValue;
  if ((ldq % 8) || (ldk % 8) || (ld_vt % 8) || (ldo % 8) || (rd > 0 && (ld_kr % 8)) || ld_vt < tokens ||
      (gate != nullptr && (ldg % 8)))
    return (int)cudaErrorInvalidValue;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)kr | (uintptr_t)vt | (uintptr_t)out | (uintptr_t)gate) & 15)
    return (int)cudaErrorInvalidValue;
  if (pool < 0 || (pool > 0 && (window < 1 || chunk > 0 || rd > 0 || kp == nullptr || vp == nullptr || pool_row == nullptr ||
                                pool_rows < 1 || (ld_kp % 8) || (ld_vp % 8) || ld_vp < pool_rows ||
                                (((uintptr_t)kp | (uintptr_t)vp) & 15))))
    return (int)cudaErrorInvalidValue;
  Args a = {};
  a.out = out; a.seq_row = seq_row; a.seq_len = seq_len; a.err = err; a.ldo = ldo;
  a.dim = dim; a.rd = rd; a.vd = vd; a.window = window;
  a.nbn = (dim + 63) / 64;
  a.nbr = (rd + 63) / 64;
  a.group = H / G;
  a.sink = sink;
  a.chunk = chunk; a.sinks = sinks; a.gate = gate; a.ldg = ldg; a.gate_scale = gate_scale;
  a.pool = pool; a.pool_row = pool_row;
  a.scale_log2 = scale * 1.4426950408889634f;
  cudaStream_t st = (cudaStream_t)stream;
  auto run = [&](auto* tag, auto dv) {
    return launch<std::remove_pointer_t<decltype(tag)>, decltype(dv)::value>(
        q, ldq, k, ldk, kr, ld_kr, vt, ld_vt, kp, ld_kp, vp, ld_vp, pool_rows, a, B, H, tokens, max_len, st);
  };
  using D64 = std::integral_constant<int, 64>;
  using D128 = std::integral_constant<int, 128>;
  if (dtype == DT_F16) return vd <= 64 ? run((__half*)nullptr, D64{}) : run((__half*)nullptr, D128{});
  return vd <= 64 ? run((__nv_bfloat16*)nullptr, D64{}) : run((__nv_bfloat16*)nullptr, D128{});
}
