// Gated linear recurrence with a short causal convolution in front of it (the recurrent block of hybrid decoders):
//
//   u_t = sum_k taps[c][k] x_{t-K+1+k} + bias[c]                        per channel, previous inputs from the state
//   log a_t = -c * sigmoid(zr_t + br) * softplus(lam),  a_t = exp(log a_t)
//   S_t = a_t S_{t-1} + sqrt(1 - a_t^2) * sigmoid(zi_t + bi) * u_t      fp32
//   out_t = S_t * gelu_tanh(y_t)
//
//   conv_state_kernel   the convolution; its result leaves as a high and a low bf16 part side by side per block of
//                       channels, so that the block-diagonal gate product (grouped tensor-core GEMM over [high | low]
//                       against [W | W]) sees 16 mantissa bits; in fp32 it is one plain value
//   lru_scan kernels    gates, decay and recurrence.  Up to one chunk of tokens: a single pass, one thread per channel.
//                       Longer inputs: pass 1 leaves every chunk's total log decay and end state, pass 2 folds the
//                       chunks before its own and runs the recurrence again from there.
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

struct ConvStateParams {
  const void* x;            // [B*S, ldx], channels at column 0
  long long ldx;
  const void* taps;         // [C, K]
  const void* bias;         // [C]
  float* state;             // [B, K - 1, C], oldest input first
  void* u;                  // bf16: [B*S, blocks, 2, C / blocks]; fp32: [B*S, C]
  int B, S, C, K, blocks;
};

constexpr int kMaxTaps = 16;

// One thread per (sequence, channel) for the first K - 1 rows (they read the state, and this thread also writes the new
// one), one thread per (row, channel) for the others.
template <typename T>
__global__ void __launch_bounds__(128) conv_state_kernel(const ConvStateParams p) {
  const int c = blockIdx.y * 128 + threadIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  if (c >= p.C) return;
  const int K = p.K, hist = K - 1;
  const int head = min(hist, p.S);
  const int units = (head > 0 ? 1 : 0) + p.S - head;      // blocks per sequence
  const int b = blockIdx.x / units, unit = blockIdx.x % units;
  const T* x = static_cast<const T*>(p.x) + (long long)b * p.S * p.ldx + c;
  const int bw = p.C / p.blocks;
  float w[kMaxTaps];
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k)
    if (k < K) w[k] = to_f32(static_cast<const T*>(p.taps)[c * K + k]);
  const float bias = to_f32(static_cast<const T*>(p.bias)[c]);
  auto put = [&](int t, float v) {
    const long long row = (long long)b * p.S + t;
    if constexpr (sizeof(T) == 2) {
      __nv_bfloat16* o = static_cast<__nv_bfloat16*>(p.u) + row * 2 * p.C + (long long)(c / bw) * 2 * bw + c % bw;
      const __nv_bfloat16 hi = __float2bfloat16(v);
      o[0] = hi;
      o[bw] = __float2bfloat16(v - __bfloat162float(hi));
    } else {
      static_cast<float*>(p.u)[row * p.C + c] = v;
    }
  };
  if (head > 0 && unit == 0) {
    float* st = p.state + (long long)b * hist * p.C + c;
    float in[2 * kMaxTaps];       // the state, then the first `head` inputs
#pragma unroll
    for (int i = 0; i < 2 * kMaxTaps; ++i) {
      if (i < hist) in[i] = st[(long long)i * p.C];
      else if (i < hist + head) in[i] = to_f32(x[(long long)(i - hist) * p.ldx]);
      else in[i] = 0.0f;
    }
#pragma unroll
    for (int t = 0; t < kMaxTaps; ++t) {
      if (t < head) {
        float acc = bias;
#pragma unroll
        for (int k = 0; k < kMaxTaps; ++k)
          if (k < K) acc = fmaf(w[k], in[t + k], acc);
        put(t, acc);
      }
    }
    for (int i = 0; i < hist; ++i) {
      const int t = p.S - hist + i;           // may lie before this call's first row: then the old state moves up
      st[(long long)i * p.C] = t >= 0 ? to_f32(x[(long long)t * p.ldx]) : st[(long long)(i + p.S) * p.C];
    }
    return;
  }
  const int t = head > 0 ? head + unit - 1 : unit;
  float acc = bias;
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k)
    if (k < K) acc = fmaf(w[k], to_f32(x[(long long)(t - hist + k) * p.ldx]), acc);
  put(t, acc);
}

struct LruParams {
  const void* u;            // as written by conv_state_kernel
  const float* z;           // [B*S, blocks, 2, C / blocks] gate products without bias: recurrence gate, input gate
  const void* br;           // [C]
  const void* bi;           // [C]
  const void* lam;          // [C]
  const void* y;            // [B*S, ldy]
  long long ldy;
  float* state;             // [B, C]
  void* out;                // [B*S, C]
  float* agg;               // [B, chunks + 1, 2, C]: log decay and end state per chunk; the last entry holds S_0
  int B, S, C, blocks, chunk, chunks;
  float c;
};

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename T>
struct LruChannel {
  const T* u;
  const float* z;
  float br, bi, decay;      // decay = -c * softplus(lam)
  int bw, C;
  __device__ __forceinline__ LruChannel(const LruParams& p, int b, int ch) {
    bw = p.C / p.blocks;
    C = p.C;
    const long long off = (long long)(ch / bw) * 2 * bw + ch % bw;
    const long long row0 = (long long)b * p.S;
    z = p.z + row0 * 2 * C + off;
    u = static_cast<const T*>(p.u) + (sizeof(T) == 2 ? row0 * 2 * C + off : row0 * C + ch);
    br = to_f32(static_cast<const T*>(p.br)[ch]);
    bi = to_f32(static_cast<const T*>(p.bi)[ch]);
    decay = -p.c * softplus_f(to_f32(static_cast<const T*>(p.lam)[ch]));
  }
  // Applies token t to S; returns its log decay.  With e = a - 1 = expm1(log a), which keeps its relative precision where
  // a is next to 1:  1 - a^2 = -e (2 + e)  and  a S = S + e S, so long memories do not drift.
  __device__ __forceinline__ float step(int t, float& S) const {
    const float* zt = z + (long long)t * 2 * C;
    float uv;
    if constexpr (sizeof(T) == 2) {
      const T* ut = u + (long long)t * 2 * C;
      uv = to_f32(ut[0]) + to_f32(ut[bw]);
    } else {
      uv = to_f32(u[(long long)t * C]);
    }
    const float log_a = decay * sigmoid_f(zt[0] + br);
    const float e = expm1f(log_a);
    S += fmaf(e, S, sqrtf(-e * (2.0f + e)) * sigmoid_f(zt[bw] + bi) * uv);
    return log_a;
  }
};

// Pass 1: chunks 0 .. chunks-2; chunk 0 starts from the state and keeps a copy of it.
template <typename T>
__global__ void __launch_bounds__(128) lru_chunk_kernel(const LruParams p) {
  const int ch = blockIdx.x * 128 + threadIdx.x, k = blockIdx.y, b = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  if (ch >= p.C) return;
  const LruChannel<T> lc(p, b, ch);
  float* agg = p.agg + (long long)b * (p.chunks + 1) * 2 * p.C + ch;
  float S = 0.0f, total = 0.0f;
  if (k == 0) {
    S = p.state[(long long)b * p.C + ch];
    agg[(long long)p.chunks * 2 * p.C] = S;
  }
  const int t0 = k * p.chunk, t1 = t0 + p.chunk;
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    total += lc.step(t, S);
  }
  agg[(long long)k * 2 * p.C] = total;
  agg[((long long)k * 2 + 1) * p.C] = S;
}

// Pass 2 (or the only pass when chunks == 1).
template <typename T>
__global__ void __launch_bounds__(128) lru_scan_kernel(const LruParams p) {
  const int ch = blockIdx.x * 128 + threadIdx.x, k = blockIdx.y, b = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  if (ch >= p.C) return;
  const LruChannel<T> lc(p, b, ch);
  float S;
  if (p.chunks == 1) {
    S = p.state[(long long)b * p.C + ch];
  } else {
    const float* agg = p.agg + (long long)b * (p.chunks + 1) * 2 * p.C + ch;
    if (k == 0) {
      S = agg[(long long)p.chunks * 2 * p.C];
    } else {
      S = agg[p.C];
#pragma unroll 4
      for (int j = 1; j < k; ++j)
        S += fmaf(expm1f(agg[(long long)j * 2 * p.C]), S, agg[((long long)j * 2 + 1) * p.C]);
    }
  }
  const int t0 = k * p.chunk, t1 = min(p.S, t0 + p.chunk);
  const T* y = static_cast<const T*>(p.y) + (long long)b * p.S * p.ldy + ch;
  T* out = static_cast<T*>(p.out) + (long long)b * p.S * p.C + ch;
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    lc.step(t, S);
    out[(long long)t * p.C] = from_f32<T>(S * gelu_tanh_f(to_f32(y[(long long)t * p.ldy])));
  }
  if (k == p.chunks - 1) p.state[(long long)b * p.C + ch] = S;
}

}  // namespace dptb

using namespace dptb;

struct DptbRecurrentArgs {
  const void* x; const void* taps; const void* conv_bias; float* conv_state; void* u;     // convolution
  const float* z; const void* br; const void* bi; const void* lam; const void* y;         // recurrence
  float* state; void* out; float* agg;
  long long ldx, ldy, agg_floats;
  int B, S, C, K, blocks, chunk, f32;
  float c;
};

extern "C" int dptb_conv_state(const DptbRecurrentArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->S <= 0) return 0;
  if (a->C <= 0 || a->K < 1 || a->K > kMaxTaps || a->blocks < 1 || a->C % a->blocks || a->ldx < a->C) return kErrBadShape;
  ConvStateParams p;
  p.x = a->x; p.ldx = a->ldx; p.taps = a->taps; p.bias = a->conv_bias; p.state = a->conv_state; p.u = a->u;
  p.B = a->B; p.S = a->S; p.C = a->C; p.K = a->K; p.blocks = a->blocks;
  const int head = a->K - 1 < a->S ? a->K - 1 : a->S;
  const long long units = ((head > 0 ? 1 : 0) + a->S - head) * (long long)a->B;
  const unsigned cy = (a->C + 127) / 128;
  if (units > 0x7fffffff || cy > 65535) return kErrTooLarge;
  const dim3 grid((unsigned)units, cy);
  return counted(1, (int)(a->f32 ? launch_k(conv_state_kernel<float>, grid, dim3(128), (size_t)0, st, p)
                                 : launch_k(conv_state_kernel<__nv_bfloat16>, grid, dim3(128), (size_t)0, st, p)));
}

extern "C" int dptb_lru_scan(const DptbRecurrentArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->S <= 0) return 0;
  if (a->C <= 0 || a->blocks < 1 || a->C % a->blocks || a->chunk < 1 || a->ldy < a->C) return kErrBadShape;
  LruParams p;
  p.u = a->u; p.z = a->z; p.br = a->br; p.bi = a->bi; p.lam = a->lam; p.y = a->y; p.ldy = a->ldy;
  p.state = a->state; p.out = a->out; p.agg = a->agg;
  p.B = a->B; p.S = a->S; p.C = a->C; p.blocks = a->blocks; p.chunk = a->chunk;
  p.chunks = (a->S + a->chunk - 1) / a->chunk; p.c = a->c;
  if (p.chunks > 65535 || a->B > 65535) return kErrTooLarge;
  const unsigned gx = (a->C + 127) / 128;
  if (p.chunks > 1) {
    if (!a->agg || a->agg_floats < (long long)a->B * (p.chunks + 1) * 2 * a->C) return kErrTooLarge;
    const dim3 g1(gx, p.chunks - 1, a->B);
    const int rc = counted(1, (int)(a->f32 ? launch_k(lru_chunk_kernel<float>, g1, dim3(128), (size_t)0, st, p)
                                           : launch_k(lru_chunk_kernel<__nv_bfloat16>, g1, dim3(128), (size_t)0, st, p)));
    if (rc) return rc;
  }
  const dim3 g2(gx, p.chunks, a->B);
  return counted(1, (int)(a->f32 ? launch_k(lru_scan_kernel<float>, g2, dim3(128), (size_t)0, st, p)
                                 : launch_k(lru_scan_kernel<__nv_bfloat16>, g2, dim3(128), (size_t)0, st, p)));
}
