// Dropless mixture of experts on one GPU: routing and the permutation of token rows into expert order.
//
//   moe_router_kernel   router logits (fp32 products), the `top` largest, softmax over those alone; one CTA per token
//                       (decode, and the fp32 path)
//   moe_topk_kernel     the same choice from logits a GEMM has written; one warp per token (prompts)
//   moe_place_kernel    rows in expert order: exclusive scan of the experts' counts, slot of every (token, choice), copy
//                       of the token's row there; also the row offsets the grouped GEMM reads
// The experts themselves are the grouped GEMM (gemm_grouped.cu), the weighted sum of their outputs rides in the residual
// kernel (stream_norm.cu).  Nothing is read back to the host.  The order of rows inside an expert is arbitrary; every
// row is computed by itself, so results do not depend on it.
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

constexpr int kMoeMaxExperts = 1024;
constexpr int kMoeMaxTop = 32;

// Floats as unsigned integers of the same order, and back.
__device__ __forceinline__ uint32_t ordered_bits(float v) {
  const uint32_t u = __float_as_uint(v);
  return (u & 0x80000000u) ? ~u : u | 0x80000000u;
}
__device__ __forceinline__ float from_ordered(uint32_t k) {
  return __uint_as_float((k & 0x80000000u) ? k & 0x7fffffffu : ~k);
}

// One warp chooses the `top` largest of `sel` (shared memory, E values, consumed).  Ties resolve to the lowest index.  A
// lane keeps the best of its own experts (lane, lane + 32, ...); a round is two warp reductions, and only the winner's
// lane looks through its experts again.
__device__ __forceinline__ void choose_top(float* sel, int E, int top, int lane, int* idx, float* w, int* count) {
  constexpr uint32_t kNone = 0xffffffffu;
  auto best = [&](uint32_t& key, uint32_t& at) {
    key = 0;
    at = kNone;
    for (int e = lane; e < E; e += 32) {
      const uint32_t k = ordered_bits(sel[e]);
      if (at == kNone || k > key) {
        key = k;
        at = e;
      }
    }
  };
  uint32_t key, at;
  best(key, at);
  float mine = 0.0f, first = 0.0f, sum = 0.0f;
  for (int j = 0; j < top; ++j) {
    const uint32_t k = __reduce_max_sync(0xffffffffu, key);
    const uint32_t e = __reduce_min_sync(0xffffffffu, key == k ? at : kNone);
    const float v = from_ordered(k);
    if (j == 0) first = v;
    const float ex = expf(v - first);
    sum += ex;
    if (lane == j) mine = ex;
    if (at == e) {
      idx[j] = (int)e;
      sel[e] = -INFINITY;
      atomicAdd(&count[e], 1);
      best(key, at);
    }
  }
  if (lane < top) w[lane] = mine / sum;
}

constexpr int kRouterThreads = 512;

template <typename T>
__global__ void __launch_bounds__(kRouterThreads)
moe_router_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ router, int D, int E, int top, int* idx,
                  float* w, int* count) {
  extern __shared__ __align__(16) float sm[];       // [D] the token, [E] logits
  float* logit = sm + D;
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int kWarps = kRouterThreads / 32, kAtOnce = 4;      // a warp works on four experts at a time
  pdl_wait();
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < D; i += kRouterThreads) sm[i] = to_f32(x[(long long)t * ldx + i]);
  __syncthreads();
  for (int e0 = warp; e0 < E; e0 += kWarps * kAtOnce) {
    float acc[kAtOnce];
    const T* r[kAtOnce];
#pragma unroll
    for (int q = 0; q < kAtOnce; ++q) {
      acc[q] = 0.0f;
      r[q] = router + (long long)min(e0 + q * kWarps, E - 1) * D;
    }
    if (D % 8 == 0) {
#pragma unroll 2
      for (int i = lane * 8; i < D; i += 256) {
        Raw8<T> raw[kAtOnce];
#pragma unroll
        for (int q = 0; q < kAtOnce; ++q) raw[q].load(r[q] + i);
        float xv[8];
        Vec8<float>::load(sm + i, xv);
#pragma unroll
        for (int q = 0; q < kAtOnce; ++q) {
          float v[8];
          raw[q].unpack(v);
#pragma unroll
          for (int k = 0; k < 8; ++k) acc[q] = fmaf(v[k], xv[k], acc[q]);
        }
      }
    } else {
      for (int i = lane; i < D; i += 32)
#pragma unroll
        for (int q = 0; q < kAtOnce; ++q) acc[q] = fmaf(to_f32(r[q][i]), sm[i], acc[q]);
    }
#pragma unroll
    for (int q = 0; q < kAtOnce; ++q) {
      const float z = warp_sum(acc[q]);
      if (lane == 0 && e0 + q * kWarps < E) logit[e0 + q * kWarps] = z;
    }
  }
  __syncthreads();
  if (warp == 0) choose_top(logit, E, top, lane, idx + (long long)t * top, w + (long long)t * top, count);
}

constexpr int kTopkTokens = 32;       // per CTA, so that a count costs one global atomic per CTA and expert

__global__ void __launch_bounds__(256)
moe_topk_kernel(const float* __restrict__ logits, long long ld, int T_, int E, int top, int* idx, float* w, int* count) {
  extern __shared__ __align__(16) float sm[];       // [8][E] logits, [E] counts
  int* hist = reinterpret_cast<int*>(sm + 8 * E);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int e = threadIdx.x; e < E; e += 256) hist[e] = 0;
  pdl_wait();
  pdl_launch_dependents();
  __syncthreads();
  float* sel = sm + warp * E;
  for (int i = warp; i < kTopkTokens; i += 8) {
    const long long t = (long long)blockIdx.x * kTopkTokens + i;
    if (t >= T_) break;
    for (int e = lane; e < E; e += 32) sel[e] = logits[t * ld + e];
    __syncwarp();
    choose_top(sel, E, top, lane, idx + t * top, w + t * top, hist);
    __syncwarp();
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256)
    if (hist[e]) atomicAdd(&count[e], hist[e]);
}

constexpr int kPlacePairs = 32;

template <typename T>
__global__ void __launch_bounds__(256)
moe_place_kernel(const T* __restrict__ x, long long ldx, const int* __restrict__ idx, const int* __restrict__ count,
                 int* cursor, int* offsets, int* slot, T* xs, int pairs, int top, int E, int D) {
  __shared__ int off[kMoeMaxExperts + 1];
  __shared__ int hist[kMoeMaxExperts];
  __shared__ int pair_slot[kPlacePairs];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  pdl_launch_dependents();
  for (int e = threadIdx.x; e < E; e += 256) hist[e] = 0;
  if (warp == 0) {
    int carry = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int n = e0 + lane < E ? count[e0 + lane] : 0;
      int inc = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += v;
      }
      if (e0 + lane < E) off[e0 + lane] = carry + inc - n;
      carry += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (lane == 0) off[E] = carry;
  }
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e <= E; e += 256) offsets[e] = off[e];
  const int p0 = blockIdx.x * kPlacePairs;
  int rank = 0, ex = 0;
  const bool mine = threadIdx.x < kPlacePairs && p0 + (int)threadIdx.x < pairs;
  if (mine) {
    ex = idx[p0 + threadIdx.x];
    rank = atomicAdd(&hist[ex], 1);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256) {
    const int n = hist[e];
    if (n > 0) hist[e] = atomicAdd(&cursor[e], n);     // first place of this block's rows inside the expert
  }
  __syncthreads();
  if (mine) {
    const int s = off[ex] + hist[ex] + rank;
    pair_slot[threadIdx.x] = s;
    slot[p0 + threadIdx.x] = s;
  }
  __syncthreads();
  for (int i = warp; i < kPlacePairs; i += 8) {
    if (p0 + i >= pairs) break;
    const T* src = x + (long long)((p0 + i) / top) * ldx;
    T* dst = xs + (long long)pair_slot[i] * D;
    constexpr int kVec = 16 / sizeof(T);
    if (D % kVec == 0 && ldx % kVec == 0) {
      for (int v = lane; v < D / kVec; v += 32)
        reinterpret_cast<uint4*>(dst)[v] = reinterpret_cast<const uint4*>(src)[v];
    } else {
      for (int v = lane; v < D; v += 32) dst[v] = src[v];
    }
  }
}

}  // namespace dptb

using namespace dptb;

struct DptbMoeArgs {
  const void* x; const void* router; const float* logits;
  int* idx; float* w; int* count; int* cursor; int* offsets; int* slot; void* xs;
  long long ldx, ld_logits;
  int T, D, E, top, f32;
};

extern "C" int dptb_moe_router(const DptbMoeArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->T <= 0) return 0;
  if (a->E < 1 || a->E > kMoeMaxExperts || a->top < 1 || a->top > kMoeMaxTop || a->top > a->E || a->D < 1) return kErrBadShape;
  if (a->logits) {
    return counted(1, (int)launch_k(moe_topk_kernel, dim3((a->T + kTopkTokens - 1) / kTopkTokens), dim3(256), (size_t)9 * a->E * 4, st, a->logits,
                                    a->ld_logits, a->T, a->E, a->top, a->idx, a->w, a->count));
  }
  const size_t bytes = (size_t)(a->D + a->E) * 4;
  if (bytes > 48 * 1024) return kErrTooLarge;
  if (a->D % 8 == 0 && (reinterpret_cast<uintptr_t>(a->router) & 15)) return kErrBadShape;
  if (a->f32)
    return counted(1, (int)launch_k(moe_router_kernel<float>, dim3(a->T), dim3(kRouterThreads), bytes, st, (const float*)a->x, a->ldx,
                                    (const float*)a->router, a->D, a->E, a->top, a->idx, a->w, a->count));
  return counted(1, (int)launch_k(moe_router_kernel<__nv_bfloat16>, dim3(a->T), dim3(kRouterThreads), bytes, st,
                                  (const __nv_bfloat16*)a->x, a->ldx, (const __nv_bfloat16*)a->router, a->D, a->E, a->top,
                                  a->idx, a->w, a->count));
}

extern "C" int dptb_moe_place(const DptbMoeArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  const int pairs = a->T * a->top;
  if (pairs <= 0) return 0;
  if (a->E < 1 || a->E > kMoeMaxExperts || a->D < 1 || (reinterpret_cast<uintptr_t>(a->x) & 15) ||
      (reinterpret_cast<uintptr_t>(a->xs) & 15))
    return kErrBadShape;
  const dim3 grid((pairs + kPlacePairs - 1) / kPlacePairs);
  if (a->f32)
    return counted(1, (int)launch_k(moe_place_kernel<float>, grid, dim3(256), (size_t)0, st, (const float*)a->x, a->ldx,
                                    (const int*)a->idx, (const int*)a->count, a->cursor, a->offsets, a->slot,
                                    (float*)a->xs, pairs, a->top, a->E, a->D));
  return counted(1, (int)launch_k(moe_place_kernel<__nv_bfloat16>, grid, dim3(256), (size_t)0, st,
                                  (const __nv_bfloat16*)a->x, a->ldx, (const int*)a->idx, (const int*)a->count, a->cursor,
                                  a->offsets, a->slot, (__nv_bfloat16*)a->xs, pairs, a->top, a->E, a->D));
}
