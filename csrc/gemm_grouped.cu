// Grouped GEMM on tcgen05 tensor cores:  out_g = act(x_g W_g^T)  for many groups in one persistent launch.
//
// Two kinds of groups, chosen per segment:
//   rows  (offsets != null)  group g owns the token rows [offsets[g], offsets[g+1]) of x (device memory, so nothing is
//                            read back to the host): a mixture of experts whose rows are sorted by expert
//   cols  (offsets == null)  every group owns all M rows and the columns [g * x_col_stride, + K) of x, and writes the
//                            columns [g * out_col_stride, + N) of out: block-diagonal and per-head products
// A launch takes up to two segments with sizes of their own (routed experts plus a shared one).
//
// The weight is the M = 128 side of the tensor core and the tokens are the N side, so the token tile can be as narrow as
// the work is: BN = 32 or 64 while decoding (a tile is then a stream of weights), 128 or 256 in prompts.
//   warp 0      TMA producer: 128 x 64 weight and BN x 64 token tiles through a ring
//   warp 1      tcgen05.mma issuer, two accumulators in TMEM
//   warps 2-9   epilogue: a lane owns one weight row = one output feature; neighbouring lanes exchange tokens so that
//               bf16 results leave as pairs of features, 64 contiguous bytes per row and warp
// Any other shape, alignment or fp32 input runs the SIMT kernel below.
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

constexpr int kGgBM = 128, kGgBK = 64;
constexpr int kGgThreads = 320;
constexpr int kGgMaxGroups = 1024;   // over both segments

struct GroupedSeg {
  int groups, N, K, M;
  int x_col_stride, out_col_stride;
  const int* offsets;
  void* out;
  long long ldc;
  int act, out_f32;
  // SIMT path only
  const void* x;
  const void* w;
  long long ldx, ldw;
};
struct GroupedParams {
  GroupedSeg seg[2];
  int nseg;
};

__device__ __forceinline__ float grouped_act(float v, int act) {
  if (act == 1) {
    v = fmaxf(v, 0.0f);
    return v * v;
  }
  return v;
}

template <int BN, int STAGES>
struct GroupedSmem {
  static constexpr int kWBytes = kGgBM * kGgBK * 2;
  static constexpr int kXBytes = BN * kGgBK * 2;
  static constexpr int kStage = kWBytes + kXBytes;
  static constexpr int kBarOff = STAGES * kStage;
  static constexpr int kPrefixOff = kBarOff + (2 * STAGES + 5) * 8 + 24;
  static constexpr int kTotal = kPrefixOff + (kGgMaxGroups + 3) * 4 + 1024;
  static_assert(kTotal <= 227 * 1024, "grouped GEMM: shared memory budget");
};

// Which group, weight tile and token tile a work unit is.
struct GroupedTile {
  int seg, g, n0, row0, row_end, num_kb;
};
template <int BN>
__device__ __forceinline__ GroupedTile grouped_tile(const GroupedParams& p, const int* prefix, int total_groups, int t) {
  int lo = 0, hi = total_groups - 1;      // last group whose first tile is <= t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (prefix[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  GroupedTile r;
  r.seg = (p.nseg > 1 && lo >= p.seg[0].groups) ? 1 : 0;
  const GroupedSeg& s = p.seg[r.seg];
  r.g = lo - (r.seg ? p.seg[0].groups : 0);
  const int begin = s.offsets ? s.offsets[r.g] : 0;
  r.row_end = s.offsets ? s.offsets[r.g + 1] : s.M;
  const int tt_n = (r.row_end - begin + BN - 1) / BN;
  const int local = t - prefix[lo];
  r.n0 = (local / tt_n) * kGgBM;          // token tiles of one weight tile are neighbours: the weights stay in L2
  r.row0 = begin + (local % tt_n) * BN;
  r.num_kb = (s.K + kGgBK - 1) / kGgBK;
  return r;
}

template <int BN, int STAGES>
__global__ void __launch_bounds__(kGgThreads, 1)
gemm_grouped_kernel(const __grid_constant__ CUtensorMap tmW0, const __grid_constant__ CUtensorMap tmX0,
                    const __grid_constant__ CUtensorMap tmW1, const __grid_constant__ CUtensorMap tmX1,
                    const GroupedParams p) {
  using L = GroupedSmem<BN, STAGES>;
  constexpr int TMEM_COLS = 2 * BN;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + L::kBarOff);
  uint64_t* empty_bar = full_bar + STAGES;
  uint64_t* acc_full = empty_bar + STAGES;    // [2]
  uint64_t* acc_empty = acc_full + 2;         // [2]
  uint64_t* drain_bar = acc_empty + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(drain_bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* prefix = reinterpret_cast<int*>(smem + L::kPrefixOff);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int total_groups = p.seg[0].groups + (p.nseg > 1 ? p.seg[1].groups : 0);

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    tma_prefetch_desc(&tmW0);
    tma_prefetch_desc(&tmX0);
    if (p.nseg > 1) {
      tma_prefetch_desc(&tmW1);
      tma_prefetch_desc(&tmX1);
    }
  }
  if (warp == 1) {
    if (lane == 0) {
      for (int s = 0; s < STAGES; ++s) {
        mbar_init(&full_bar[s], 1);
        mbar_init(&empty_bar[s], 1);
      }
      for (int a = 0; a < 2; ++a) {
        mbar_init(&acc_full[a], 1);
        mbar_init(&acc_empty[a], 8);
      }
      mbar_init(drain_bar, 1);
      mbar_fence_init();
    }
    __syncwarp();
    tmem_alloc<TMEM_COLS>(tmem_slot);
  }
  pdl_wait();
  pdl_launch_dependents();
  if (warp == 0) {
    // first tile of every group: exclusive scan over the groups' tile counts
    int carry = 0;
    for (int g0 = 0; g0 < total_groups; g0 += 32) {
      const int gi = g0 + lane;
      int n = 0;
      if (gi < total_groups) {
        const int sg = (p.nseg > 1 && gi >= p.seg[0].groups) ? 1 : 0;
        const GroupedSeg& s = p.seg[sg];
        const int g = gi - (sg ? p.seg[0].groups : 0);
        const int cnt = s.offsets ? s.offsets[g + 1] - s.offsets[g] : s.M;
        n = ((cnt + BN - 1) / BN) * ((s.N + kGgBM - 1) / kGgBM);
      }
      int inc = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += v;
      }
      if (gi < total_groups) prefix[gi] = carry + inc - n;
      carry += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (lane == 0) prefix[total_groups] = carry;
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  const int total_tiles = prefix[total_groups];

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      int issued = 0;
      bool ok = true;
      for (int t = blockIdx.x; t < total_tiles && ok; t += gridDim.x) {
        const GroupedTile tl = grouped_tile<BN>(p, prefix, total_groups, t);
        const GroupedSeg& s = p.seg[tl.seg];
        const CUtensorMap* tw = tl.seg ? &tmW1 : &tmW0;
        const CUtensorMap* tx = tl.seg ? &tmX1 : &tmX0;
        const int xc0 = s.offsets ? 0 : tl.g * s.x_col_stride;
        const int wrow = tl.g * s.N + tl.n0;
        for (int kb = 0; kb < tl.num_kb; ++kb, ++issued) {
          const int st = issued % STAGES;
          if (!mbar_wait(&empty_bar[st], ((issued / STAGES) & 1) ^ 1, abort_flag, kWaitEmptyTimeout)) {
            ok = false;
            break;
          }
          mbar_arrive_expect_tx(&full_bar[st], L::kStage);
          uint8_t* dst = smem + st * L::kStage;
          tma_load_2d(dst, tw, &full_bar[st], kb * kGgBK, wrow);
          tma_load_2d(dst + L::kWBytes, tx, &full_bar[st], xc0 + kb * kGgBK, tl.row0);
        }
      }
      if (*abort_flag) {
        // Do not leave while a tile copy may still be writing this CTA's shared memory.
        const int n = issued < STAGES ? issued : STAGES;
        const uint64_t t0 = global_timer_ns();
        for (int j = 0; j < n; ++j) {
          const int i = issued - 1 - j;
          while (!mbar_try_wait(&full_bar[i % STAGES], (i / STAGES) & 1) &&
                 global_timer_ns() - t0 < kWaitLimitNs / 4) {}
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_bf16(kGgBM, BN, false, false);
      int consumed = 0, it = 0;
      bool ok = true, issued_any = false;
      for (int t = blockIdx.x; t < total_tiles && ok; t += gridDim.x, ++it) {
        const GroupedTile tl = grouped_tile<BN>(p, prefix, total_groups, t);
        const int acc = it & 1;
        if (!mbar_wait(&acc_empty[acc], ((it >> 1) & 1) ^ 1, abort_flag, kWaitTmemEmptyTimeout)) break;
        tc_fence_after_sync();
        for (int kb = 0; kb < tl.num_kb; ++kb, ++consumed) {
          const int st = consumed % STAGES;
          if (!mbar_wait(&full_bar[st], (consumed / STAGES) & 1, abort_flag, kWaitFullTimeout)) {
            ok = false;
            break;
          }
          tc_fence_after_sync();
          const uint32_t wa = smem_u32(smem + st * L::kStage);
          const uint32_t xa = wa + L::kWBytes;
#pragma unroll
          for (int k = 0; k < kGgBK / 16; ++k)
            umma_bf16(tmem_base + acc * BN, make_smem_desc(wa + k * 32, 16, 1024), make_smem_desc(xa + k * 32, 16, 1024),
                      idesc, (kb != 0 || k != 0) ? 1u : 0u);
          issued_any = true;
          umma_commit(&empty_bar[st]);
        }
        if (ok) umma_commit(&acc_full[acc]);
      }
      if (*abort_flag && issued_any) {
        umma_commit(drain_bar);
        const uint64_t t0 = global_timer_ns();
        while (!mbar_try_wait(drain_bar, 0) && global_timer_ns() - t0 < kWaitLimitNs / 4) {}
      }
    }
  } else {
    // ------------------------------------------------------------------ epilogue
    const int q = warp & 3;                 // TMEM lane quarter
    const int half = (warp - 2) >> 2;       // token columns [half * BN / 2, + BN / 2)
    int it = 0;
    for (int t = blockIdx.x; t < total_tiles; t += gridDim.x, ++it) {
      const GroupedTile tl = grouped_tile<BN>(p, prefix, total_groups, t);
      const GroupedSeg& s = p.seg[tl.seg];
      const int acc = it & 1;
      if (!__all_sync(0xffffffffu, mbar_wait(&acc_full[acc], (it >> 1) & 1, abort_flag, kWaitTmemFullTimeout))) break;
      tc_fence_after_sync();
      const int n = tl.n0 + q * 32 + lane;
      const long long col = (s.offsets ? 0 : (long long)tl.g * s.out_col_stride) + n;
      const bool n_ok = n < s.N;
#pragma unroll 1
      for (int c = 0; c < BN / 2; c += 16) {
        const int tok0 = tl.row0 + half * (BN / 2) + c;
        if (tok0 >= tl.row_end) break;      // the same for the whole warp
        uint32_t r[16];
        tmem_ld_32x16(tmem_base + ((uint32_t)(q * 32) << 16) + acc * BN + half * (BN / 2) + c, r);
        tmem_ld_wait();
        if (s.out_f32) {
          float* o = static_cast<float*>(s.out) + col;
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (n_ok && tok0 + i < tl.row_end) o[(long long)(tok0 + i) * s.ldc] = grouped_act(__uint_as_float(r[i]), s.act);
        } else {
          // even lanes keep token i and take their neighbour's feature n + 1; odd lanes keep token i + 1
          __nv_bfloat16* o = static_cast<__nv_bfloat16*>(s.out) + (col & ~1ll);
          const int odd = lane & 1;
#pragma unroll
          for (int i = 0; i < 16; i += 2) {
            const float a = grouped_act(__uint_as_float(r[i]), s.act), b = grouped_act(__uint_as_float(r[i + 1]), s.act);
            const float other = __shfl_xor_sync(0xffffffffu, odd ? a : b, 1);
            const uint32_t v = odd ? pack_bf16x2(other, b) : pack_bf16x2(a, other);
            const int tok = tok0 + i + odd;
            if (n_ok && tok < tl.row_end) *reinterpret_cast<uint32_t*>(o + (long long)tok * s.ldc) = v;
          }
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&acc_empty[acc]);
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc<TMEM_COLS>(tmem_base);
  }
}

// ----------------------------------------------------------------------------- SIMT kernel
// Any size, alignment and dtype: 64 x 64 tile, 4 x 4 outputs per thread, fp32 multiply-adds.
template <typename T>
__global__ void __launch_bounds__(256) gemm_grouped_simt_kernel(const GroupedSeg s) {
  __shared__ float As[16][64 + 1];
  __shared__ float Bs[16][64 + 1];
  const int g = blockIdx.z;
  const int begin = s.offsets ? s.offsets[g] : 0;
  const int end = s.offsets ? s.offsets[g + 1] : s.M;
  const int m0 = begin + blockIdx.y * 64, n0 = blockIdx.x * 64;
  if (m0 >= end) return;
  const T* x = static_cast<const T*>(s.x) + (s.offsets ? 0 : (long long)g * s.x_col_stride);
  const T* w = static_cast<const T*>(s.w) + (long long)g * s.N * s.ldw;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < s.K; k0 += 16) {
    for (int i = threadIdx.x; i < 16 * 64; i += 256) {
      const int kk = i & 15, mm = i >> 4, k = k0 + kk;
      As[kk][mm] = (m0 + mm < end && k < s.K) ? to_f32(x[(long long)(m0 + mm) * s.ldx + k]) : 0.0f;
      Bs[kk][mm] = (n0 + mm < s.N && k < s.K) ? to_f32(w[(long long)(n0 + mm) * s.ldw + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(As[kk][ty * 4 + i], Bs[kk][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
  const long long oc = s.offsets ? 0 : (long long)g * s.out_col_stride;
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= end || n >= s.N) continue;
      const float v = grouped_act(acc[i][j], s.act);
      const long long at = (long long)m * s.ldc + oc + n;
      if (s.out_f32) static_cast<float*>(s.out)[at] = v;
      else static_cast<T*>(s.out)[at] = from_f32<T>(v);
    }
}

template <int BN, int STAGES>
static int launch_grouped(const CUtensorMap* tm, const GroupedParams& p, int max_tiles, cudaStream_t st) {
  using L = GroupedSmem<BN, STAGES>;
  auto kern = gemm_grouped_kernel<BN, STAGES>;
  static bool configured = false;
  if (!configured) {
    DPTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kTotal));
    configured = true;
  }
  const int grid = max_tiles < sm_count() ? max_tiles : sm_count();
  return counted(1, (int)launch_k(kern, dim3(grid), dim3(kGgThreads), L::kTotal, st, tm[0], tm[1], tm[2], tm[3], p));
}

}  // namespace dptb

using namespace dptb;

// One segment (mirrored by a ctypes.Structure).
struct DptbGroupedSeg {
  const void* x;          // [x_rows, x_cols], row stride ldx
  const void* w;          // [groups * N, K], row stride ldw
  void* out;
  const int* offsets;     // device [groups + 1] or null
  long long ldx, ldw, ldc;
  int groups, N, K;
  int M;                  // rows of x (the capacity when offsets are given)
  int x_cols, x_col_stride, out_col_stride;
  int f32;                // x and w are fp32 (SIMT)
  int act;                // 0 none, 1 square of relu
  int out_f32;
  int rows_hint;          // rows a group is expected to have; the first segment's picks the token tile
};

extern "C" int dptb_gemm_grouped(const DptbGroupedSeg* segs, int nseg, int force_simt, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (nseg < 1 || nseg > 2) return kErrBadShape;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  bool tc = !force_simt;
  int total_groups = 0;
  GroupedParams p;
  p.nseg = nseg;
  for (int i = 0; i < nseg; ++i) {
    const DptbGroupedSeg& a = segs[i];
    if (a.groups <= 0 || a.N <= 0 || a.K <= 0 || a.M < 0) return kErrBadShape;
    if (!a.offsets && (long long)(a.groups - 1) * a.x_col_stride + a.K > a.x_cols) return kErrBadShape;
    if (a.offsets && a.K > a.x_cols) return kErrBadShape;
    if (a.ldx < a.x_cols || a.ldw < a.K) return kErrBadShape;
    if (a.f32 != segs[0].f32) return kErrUnsupported;
    total_groups += a.groups;
    // the token tile starts at a multiple of 64 columns from the group's first column: 16-byte alignment of the copy
    // needs that first column and every row stride to be multiples of 8 elements
    tc = tc && !a.f32 && al16(a.x) && al16(a.w) && a.ldx % 8 == 0 && a.ldw % 8 == 0 && (a.offsets || a.x_col_stride % 8 == 0) &&
         a.K % 8 == 0 && a.N % 2 == 0 && a.ldc % 2 == 0 && a.out_col_stride % 2 == 0 &&
         (reinterpret_cast<uintptr_t>(a.out) & 3) == 0;
    GroupedSeg& s = p.seg[i];
    s.groups = a.groups; s.N = a.N; s.K = a.K; s.M = a.M;
    s.x_col_stride = a.x_col_stride; s.out_col_stride = a.out_col_stride;
    s.offsets = a.offsets; s.out = a.out; s.ldc = a.ldc; s.act = a.act; s.out_f32 = a.out_f32;
    s.x = a.x; s.w = a.w; s.ldx = a.ldx; s.ldw = a.ldw;
  }
  if (nseg == 1) p.seg[1] = p.seg[0];
  tc = tc && total_groups <= kGgMaxGroups;
  if (!tc) {
    for (int i = 0; i < nseg; ++i) {
      const GroupedSeg& s = p.seg[i];
      if (s.M == 0) continue;
      const dim3 grid((s.N + 63) / 64, (s.M + 63) / 64, s.groups);
      if (grid.y > 65535 || grid.z > 65535) return kErrTooLarge;
      if (segs[i].f32) gemm_grouped_simt_kernel<float><<<grid, 256, 0, st>>>(s);
      else gemm_grouped_simt_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(s);
      const int rc = counted(1, (int)cudaGetLastError());
      if (rc) return rc;
    }
    return 0;
  }
  const int hint = segs[0].rows_hint;
  const int bn = hint <= 24 ? 32 : (hint <= 64 ? 64 : (hint <= 128 ? 128 : 256));
  CUtensorMap tm[4];
  long long max_tiles = 0;
  for (int i = 0; i < nseg; ++i) {
    const DptbGroupedSeg& a = segs[i];
    if (a.M == 0) return kErrBadShape;
    int rc = encode_tmap_2d_bf16(&tm[2 * i], a.w, (uint64_t)a.K, (uint64_t)a.groups * a.N, (uint64_t)a.ldw * 2, 64, kGgBM);
    if (rc) return rc;
    rc = encode_tmap_2d_bf16(&tm[2 * i + 1], a.x, (uint64_t)a.x_cols, (uint64_t)a.M, (uint64_t)a.ldx * 2, 64, (uint32_t)bn);
    if (rc) return rc;
    const long long tn = (a.N + kGgBM - 1) / kGgBM;
    const long long tt = a.offsets ? a.M / bn + (a.groups < a.M ? a.groups : a.M) : (long long)a.groups * ((a.M + bn - 1) / bn);
    max_tiles += tn * tt;
  }
  if (nseg == 1) { tm[2] = tm[0]; tm[3] = tm[1]; }
  if (max_tiles > (1 << 30)) return kErrTooLarge;
  if (bn == 32) return launch_grouped<32, 8>(tm, p, (int)max_tiles, st);
  if (bn == 64) return launch_grouped<64, 8>(tm, p, (int)max_tiles, st);
  if (bn == 128) return launch_grouped<128, 6>(tm, p, (int)max_tiles, st);
  return launch_grouped<256, 4>(tm, p, (int)max_tiles, st);
}
