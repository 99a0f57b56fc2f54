// Dense tcgen05 GEMM for decoders with a 32-bit residual stream and dense expert banks, sm_100a:
//
//     out = x[M, K] . W[N, K]^T (+ bias)  out_mode 0: 16-bit, optionally squared relu      1: added to an fp32 stream
//                                         2: fp32 (router scores, logits)
//     y = glu(row_scale * (x . W_gu^T))                    gate / up rows interleaved in 16-row tiles, N / 2 columns
//     y = gelu_tanh(gate) * up, silu(gate) * up or a       gate / up rows interleaved in 8-row tiles, N / 2 columns
//         clamped unit
//     y = gelu_tanh(x . W^T) * the token's row of a table
//
// A second matrix (w2) may ride along: its rows multiply the same x and leave as fp32 in an output of their own.
//
// With `ranges` the launch covers a whole bank of weight matrices: group e multiplies its rows
// [ranges[e][0], + ranges[e][1]) of x, read from DEVICE memory, so one launch serves all experts of a prompt and the
// host never learns the routing.  The tile list is laid out over the groups at kernel start.
//
// Layout and roles as in tcgen05_gemm.cu: weight rows on the MMA's M side (128), tokens on its N side (32..256), both
// operands K-major in the 128-byte swizzle, two accumulators in TMEM, one persistent CTA per SM; warp 0 loads, warp 1
// issues the MMAs, warps 2-5 store.  Every mbarrier wait is bounded (codes 37 loader, 38 MMA issuer, 39 epilogue).
#include "common/utils.cuh"
#include "tcgen05_common.cuh"

namespace {

using namespace tc5;

constexpr int kBM = 128, kBK = 64, kThreads = 192;

struct Args {
  void* out;
  const float* row_scale;   // [rows of x], glu only
  const int* ranges;        // [groups][2] device, or null
  int* err;
  int64_t ldo;
  int M, N, K, groups;
  int out_mode, act;        // act 1: squared relu (out_mode 0); 2: clamped gated unit of scaled rows; 3 / 4 / 5: gelu- /
                            // silu-gated / clamped unit; 6: gelu times the token's row of `mul`
  float limit, alpha;
  const void* bias;         // T [N] or null
  float* out2;              // fp32 [M, ldo2], results of the second matrix's N2 rows (0: there is none)
  int64_t ldo2;
  int N2;
  int act_from;             // act 1: columns from this one on
  const void* mul;          // act 6: T [mul_rows, ldm]
  const int64_t* ids;       // ... and its rows, [M]
  int64_t ldm, mul_rows;
};

template <int BT>
struct Cfg {
  static constexpr int kStages = BT >= 256 ? 4 : (BT >= 128 ? 6 : 8);
  static constexpr int kABytes = kBM * kBK * 2;
  static constexpr int kBBytes = BT * kBK * 2;
  static constexpr int kStageBytes = kABytes + kBBytes;
  static constexpr int kTmemCols = 2 * BT < 32 ? 32 : 2 * BT;
  static constexpr int kSmemBytes = kStages * kStageBytes + 1024 + 256;
};

struct Tile {
  int e, nb, mb, row0, rows;
};

// walks the tile list: t only grows, so the group pointer only moves forward
template <int BT>
struct Walker {
  const Args& a;
  const int* first;     // shared: first tile of every group, [groups + 1]
  int n_tiles;          // of the first matrix, then of both
  int all_tiles;
  int e = 0;
  __device__ Walker(const Args& args, const int* f)
      : a(args), first(f), n_tiles((args.N + kBM - 1) / kBM), all_tiles(n_tiles + (args.N2 + kBM - 1) / kBM) {}
  __device__ __forceinline__ bool get(int t, Tile& o) {
    if (a.ranges == nullptr) {
      const int mt = (a.M + BT - 1) / BT;
      if (t >= mt * all_tiles) return false;
      o = {0, t / mt, t % mt, 0, a.M};
      return true;
    }
    if (t >= first[a.groups]) return false;
    while (t >= first[e + 1]) ++e;
    const int rows = a.ranges[2 * e + 1], mt = (rows + BT - 1) / BT, local = t - first[e];
    o = {e, local / mt, local % mt, a.ranges[2 * e], rows};
    return true;
  }
};

template <typename T, int BT>
__global__ void __launch_bounds__(kThreads, 1)
gemm_stream_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_w2,
                   const __grid_constant__ CUtensorMap tm_x, Args a) {
  using C = Cfg<BT>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sA = smem;
  uint8_t* sB = smem + C::kStages * C::kABytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::kStages * C::kStageBytes);
  uint64_t* full = bars;
  uint64_t* empty = bars + C::kStages;
  uint64_t* acc_full = bars + 2 * C::kStages;
  uint64_t* acc_empty = acc_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* first = reinterpret_cast<int*>(smem + C::kStages * C::kStageBytes + 256);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kblocks = (a.K + kBK - 1) / kBK;

  if (threadIdx.x == 0) {
    for (int s = 0; s < C::kStages; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&acc_full[i], 1);
      mbar_init(&acc_empty[i], 4);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) tmem_alloc(tmem_slot, C::kTmemCols);
  if (warp == 2 && a.ranges != nullptr) {     // exclusive prefix of the groups' tile counts
    const int n_tiles = (a.N + kBM - 1) / kBM;
    int run = 0;
    for (int e0 = 0; e0 < a.groups; e0 += 32) {
      const int e = e0 + lane;
      const int c = e < a.groups ? (a.ranges[2 * e + 1] + BT - 1) / BT * n_tiles : 0;
      int p = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, p, o);
        if (lane >= o) p += v;
      }
      if (e < a.groups) first[e] = run + p - c;
      run += __shfl_sync(0xffffffffu, p, 31);
    }
    if (lane == 0) first[a.groups] = run;
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  Walker<BT> walk(a, first);
  Tile tl;

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tm_w);
      if (a.N2 > 0) prefetch_tmap(&tm_w2);
      prefetch_tmap(&tm_x);
      int s = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int t = blockIdx.x; ok && walk.get(t, tl); t += gridDim.x) {
        const bool second = tl.nb >= walk.n_tiles;
        const CUtensorMap* tm = second ? &tm_w2 : &tm_w;
        const int wrow = second ? (tl.nb - walk.n_tiles) * kBM : tl.e * a.N + tl.nb * kBM, xrow = tl.row0 + tl.mb * BT;
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&empty[s], ph ^ 1, abort_flag)) { ok = false; report(a.err, 37); break; }
          mbar_expect_tx(&full[s], C::kStageBytes);
          tma_load_2d(sA + s * C::kABytes, tm, kb * kBK, wrow, &full[s]);
          tma_load_2d(sB + s * C::kBBytes, &tm_x, kb * kBK, xrow, &full[s]);
          if (++s == C::kStages) { s = 0; ph ^= 1; }
        }
      }
      if (!ok)
        for (int i = 0; i < C::kStages; ++i) mbar_wait_quiet(&full[i], 0, 1 << 12);
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = make_idesc_f16<T>(kBM, BT);
      int s = 0, it = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int t = blockIdx.x; ok && walk.get(t, tl); t += gridDim.x, ++it) {
        const int acc = it & 1;
        if (!mbar_wait(&acc_empty[acc], ((it >> 1) & 1) ^ 1, abort_flag)) { report(a.err, 38); break; }
        tcgen05_fence_after();
        const uint32_t d_tmem = tmem_base + acc * BT;
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&full[s], ph, abort_flag)) { ok = false; report(a.err, 38); break; }
          tcgen05_fence_after();
          const uint64_t ad = make_desc_sw128(smem_u32(sA + s * C::kABytes));
          const uint64_t bd = make_desc_sw128(smem_u32(sB + s * C::kBBytes));
#pragma unroll
          for (int kk = 0; kk < kBK / 16; ++kk) umma_f16(d_tmem, ad + 2 * kk, bd + 2 * kk, idesc, (kb | kk) != 0);
          umma_commit(&empty[s]);
          if (++s == C::kStages) { s = 0; ph ^= 1; }
        }
        if (ok) umma_commit(&acc_full[acc]);
      }
    }
    __syncwarp();
  } else {
    const int qd = warp & 3;      // TMEM lane quarter this warp may read
    int it = 0;
    for (int t = blockIdx.x; walk.get(t, tl); t += gridDim.x, ++it) {
      const int acc = it & 1;
      if (!mbar_wait(&acc_full[acc], (it >> 1) & 1, abort_flag)) {
        if (lane == 0) report(a.err, 39);
        break;
      }
      tcgen05_fence_after();
      const bool second = tl.nb >= walk.n_tiles;
      const int n = (second ? tl.nb - walk.n_tiles : tl.nb) * kBM + qd * 32 + lane;
      const int rows = tl.rows - tl.mb * BT;                  // rows of this tile that exist
      const int64_t xrow = tl.row0 + tl.mb * BT;
#pragma unroll 1
      for (int c = 0; c < BT / 32 && c * 32 < rows; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(tmem_base + (uint32_t(qd * 32) << 16) + acc * BT + c * 32, v);
        const int lim = min(32, rows - c * 32);
        const int64_t r0 = xrow + c * 32;
        if (second) {
          if (n < a.N2) {
            float* out = a.out2 + r0 * a.ldo2 + n;
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (j < lim) out[(int64_t)j * a.ldo2] = __uint_as_float(v[j]);
          }
          continue;
        }
        const float bn = a.bias != nullptr && n < a.N ? to_float<T>(reinterpret_cast<const T*>(a.bias)[n]) : 0.f;
        if (a.act >= 3 && a.act <= 5) {
          // lanes with bit 3 clear hold gate rows, the lanes eight above them the matching up rows: the former finish
          // the even tokens of a pair, the latter the odd ones
          const int n_out = (tl.nb * kBM + qd * 32) / 2 + (lane >> 4) * 8 + (lane & 7);
          const bool upper = lane & 8, writer = n_out < a.N / 2;
          T* out = reinterpret_cast<T*>(a.out) + (r0 + upper) * a.ldo + n_out;
#pragma unroll
          for (int j = 0; j < 32; j += 2) {
            const float s0 = __uint_as_float(v[j]) + bn, s1 = __uint_as_float(v[j + 1]) + bn;
            const float got = __shfl_xor_sync(0xffffffffu, upper ? s0 : s1, 8);
            const float gv = upper ? got : s0, uv = upper ? s1 : got;
            float f;
            if (a.act == 5) {
              const float gc = fminf(gv, a.limit);
              f = __fdividef(gc, 1.0f + __expf(-a.alpha * gc)) * (fminf(fmaxf(uv, -a.limit), a.limit) + 1.0f);
            } else {
              const float e = a.act == 4 ? gv : 1.5957691216057308f * (gv + 0.044715f * gv * gv * gv);
              f = __fdividef(gv, 1.0f + __expf(-e)) * uv;
            }
            if (writer && j + upper < lim) out[(int64_t)j * a.ldo] = from_float<T>(f);
          }
        } else if (a.act == 2) {
          // lanes 0..15 hold gate rows, lanes 16..31 the matching up rows
          const int n_out = (tl.nb * kBM + qd * 32) / 2 + (lane & 15);
          T* out = reinterpret_cast<T*>(a.out) + r0 * a.ldo + n_out;
          const bool writer = lane < 16 && n_out < a.N / 2;
          const float ws = lane < lim ? a.row_scale[r0 + lane] : 0.f;
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const float sv = __uint_as_float(v[j]) * __shfl_sync(0xffffffffu, ws, j);
            const float u = fminf(fmaxf(__shfl_down_sync(0xffffffffu, sv, 16), -a.limit), a.limit);
            const float g = fminf(sv, a.limit);
            if (writer && j < lim)
              out[(int64_t)j * a.ldo] = from_float<T>(g / (1.0f + __expf(-a.alpha * g)) * (u + 1.0f));
          }
        } else if (a.act == 6) {
          // a lane looks up one token's row for the whole warp; all loads before the first store
          const int64_t id = a.ids[r0 + min(lane, lim - 1)], row = id < 0 ? 0 : id >= a.mul_rows ? a.mul_rows - 1 : id;
          const T* mul = reinterpret_cast<const T*>(a.mul) + min(n, a.N - 1);
          T* out = reinterpret_cast<T*>(a.out) + r0 * a.ldo + n;
          T e[32];
#pragma unroll
          for (int j = 0; j < 32; ++j) e[j] = mul[__shfl_sync(0xffffffffu, row, j) * a.ldm];
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const float z = __uint_as_float(v[j]) + bn, y = 1.5957691216057308f * (z + 0.044715f * z * z * z);
            if (n < a.N && j < lim)
              out[(int64_t)j * a.ldo] = from_float<T>(__fdividef(z, 1.0f + __expf(-y)) * to_float<T>(e[j]));
          }
        } else if (n < a.N) {
          if (a.out_mode == 0) {
            T* out = reinterpret_cast<T*>(a.out) + r0 * a.ldo + n;
#pragma unroll
            for (int j = 0; j < 32; ++j) {
              float f = __uint_as_float(v[j]) + bn;
              if (a.act == 1 && n >= a.act_from) f = f > 0.f ? f * f : 0.f;
              if (j < lim) out[(int64_t)j * a.ldo] = from_float<T>(f);
            }
          } else {
            float* out = reinterpret_cast<float*>(a.out) + r0 * a.ldo + n;
            if (a.out_mode == 1) {
              float old[32];                 // all loads before the first store: one latency, not 32
#pragma unroll
              for (int j = 0; j < 32; ++j) old[j] = j < lim ? out[(int64_t)j * a.ldo] : 0.f;
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (j < lim) out[(int64_t)j * a.ldo] = old[j] + (__uint_as_float(v[j]) + bn);
            } else {
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (j < lim) out[(int64_t)j * a.ldo] = __uint_as_float(v[j]) + bn;
            }
          }
        }
      }
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&acc_empty[acc]);
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_base, C::kTmemCols);
  }
}

int sm_count() {
  int dev = 0, sms = 148;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  return sms;
}

template <typename T, int BT>
int launch(const void* x, int64_t ldx, int x_rows, const void* w, int64_t ldw, const void* w2, const Args& a,
           cudaStream_t st) {
  const CUtensorMapDataType dt =
      std::is_same<T, __half>::value ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  CUtensorMap tw, tw2, tx;
  if (!encode_2d_sw128(&tw, dt, w, (uint64_t)a.K, (uint64_t)a.N * a.groups, (uint64_t)ldw * 2, kBK, kBM)) return -1;
  if (!encode_2d_sw128(&tx, dt, x, (uint64_t)a.K, (uint64_t)x_rows, (uint64_t)ldx * 2, kBK, BT)) return -1;
  tw2 = tw;
  if (a.N2 > 0 && !encode_2d_sw128(&tw2, dt, w2, (uint64_t)a.K, (uint64_t)a.N2, (uint64_t)ldw * 2, kBK, kBM)) return -1;
  auto kern = gemm_stream_kernel<T, BT>;
  const int smem = Cfg<BT>::kSmemBytes + (a.ranges != nullptr ? (a.groups + 1) * 4 : 0);
  if (smem > 227 * 1024) return (int)cudaErrorInvalidValue;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return (int)e;
  const int64_t mt = (a.M + BT - 1) / BT + (a.ranges != nullptr ? a.groups : 0);    // upper bound of the tile count
  const int64_t tiles = mt * ((a.N + kBM - 1) / kBM + (a.N2 + kBM - 1) / kBM);
  const int sms = sm_count();
  kern<<<tiles < sms ? (int)tiles : sms, kThreads, smem, st>>>(tw, tw2, tx, a);
  return (int)cudaGetLastError();
}

template <typename T>
int dispatch(int bt, const void* x, int64_t ldx, int x_rows, const void* w, int64_t ldw, const void* w2, const Args& a,
             cudaStream_t st) {
  switch (bt) {
    case 32: return launch<T, 32>(x, ldx, x_rows, w, ldw, w2, a, st);
    case 64: return launch<T, 64>(x, ldx, x_rows, w, ldw, w2, a, st);
    case 128: return launch<T, 128>(x, ldx, x_rows, w, ldw, w2, a, st);
    case 256: return launch<T, 256>(x, ldx, x_rows, w, ldw, w2, a, st);
    default: return (int)cudaErrorInvalidValue;
  }
}

}  // namespace

// See the head of this file.  M: rows of x; with `ranges` the groups' rows partition them.  w: [groups * N, K].  bt:
// token tile (32 / 64 / 128 / 256).  row_scale only with act 2 (then out_mode 0 and N a multiple of 32).  act 1: columns from
// act_from on.  act 3 to 5: out_mode 0, N a multiple of 16.  act 6: out_mode 0, no ranges, `mul` [mul_rows, ldm] and the
// tokens' rows of it, ids [M].  bias (may be null) has N entries of the operands' type; not with act 2 or ranges.
// w2 / out2 (N2 = 0: none): N2 more rows of the same row stride, results in fp32; not with ranges or act 2.
// Strides of x and w multiples of 8 elements, bases 16-byte aligned.  Returns a cudaError_t, or -1 when the
// tensor-map encoder rejects the operands.
IPEX_API int ipex_gemm_stream(const void* x, int64_t ldx, const void* w, int64_t ldw, void* out, int64_t ldo,
                              const void* bias, const void* w2, int N2, float* out2, int64_t ldo2, const float* row_scale, const int* ranges, int groups, int M, int N, int K, int out_mode,
                              int act, float limit, float alpha, int act_from, const void* mul, int64_t ldm, int64_t mul_rows,
                              const int64_t* ids, int bt, int dtype, int* err, void* stream) {
  if (M < 1 || N < 1 || K < 1 || groups < 1 || (ldx % 8) != 0 || (ldw % 8) != 0 || out_mode < 0 || out_mode > 2)
    return (int)cudaErrorInvalidValue;
  if ((groups > 1) != (ranges != nullptr) && ranges == nullptr) return (int)cudaErrorInvalidValue;
  if (act == 2 && (row_scale == nullptr || out_mode != 0 || (N % 32) != 0)) return (int)cudaErrorInvalidValue;
  if (act < 0 || act > 6 || (act == 1 && out_mode != 0) || (act >= 3 && act <= 5 && (out_mode != 0 || (N % 16) != 0)) ||
      (act == 6 && (out_mode != 0 || ranges != nullptr || mul == nullptr || ids == nullptr || mul_rows < 1)) ||
      (bias != nullptr && (act == 2 || ranges != nullptr)))
    return (int)cudaErrorInvalidValue;
  if ((reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(w) & 15)) return (int)cudaErrorInvalidValue;
  if ((int64_t)groups * N > 0x7fffffff) return (int)cudaErrorInvalidValue;
  if (N2 < 0 || (N2 > 0 && (w2 == nullptr || out2 == nullptr || ranges != nullptr || act == 2 ||
                            (reinterpret_cast<uintptr_t>(w2) & 15))))
    return (int)cudaErrorInvalidValue;
  Args a = {out, row_scale, ranges, err, ldo, M, N, K, groups, out_mode, act, limit, alpha, bias,
            out2, ldo2, N2, act_from, mul, ids, ldm, mul_rows};
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == DT_F16) return dispatch<__half>(bt, x, ldx, M, w, ldw, w2, a, st);
  if (dtype == DT_BF16) return dispatch<__nv_bfloat16>(bt, x, ldx, M, w, ldw, w2, a, st);
  return (int)cudaErrorInvalidValue;
}
