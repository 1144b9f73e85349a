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
//   lru_scan kernels    gates, decay and recurrence, a thread per channel (or two).  Up to one chunk of tokens: a single
//                       pass.  Longer inputs: pass 1 runs every chunk from a zero state and replaces the gate products
//                       by the log decay since the chunk's start and that local state; pass 2 folds the ends of the
//                       chunks before its own into the state it starts from and adds its decayed rest to every token.
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

// Eight channels per thread, runs of kConvRun rows, up to four taps, the window in registers.
constexpr int kConvRun = 8;
__global__ void __launch_bounds__(128) conv_state_vec_kernel(const ConvStateParams p) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * 8;
  const int runs = (p.S + kConvRun - 1) / kConvRun;
  const int b = blockIdx.x / runs, t0 = (blockIdx.x % runs) * kConvRun;
  pdl_wait();
  pdl_launch_dependents();
  if (c >= p.C) return;
  const int K = p.K, hist = K - 1;
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(p.x) + (long long)b * p.S * p.ldx + c;
  const __nv_bfloat16* taps = static_cast<const __nv_bfloat16*>(p.taps) + (long long)c * K;
  float w[4][8], win[4][8], bias[8];      // tap 3 is the current row's; win[3] the current row
#pragma unroll
  for (int k = 0; k < 4; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) w[k][e] = k >= 4 - K ? __bfloat162float(taps[e * K + k - (4 - K)]) : 0.0f;
  Vec8<__nv_bfloat16>::load(static_cast<const __nv_bfloat16*>(p.bias) + c, bias);
  float* st = p.state + (long long)b * hist * p.C + c;
#pragma unroll
  for (int i = 0; i < 3; ++i) {           // the three rows before t0
    const int t = t0 - 3 + i, s = t + hist;
#pragma unroll
    for (int e = 0; e < 8; ++e) win[i][e] = 0.0f;
    if (t >= 0) Vec8<__nv_bfloat16>::load(x + (long long)t * p.ldx, win[i]);
    else if (s >= 0) Vec8<float>::load(st + (long long)s * p.C, win[i]);
  }
  if (t0 == 0 && hist > 0) {              // the only thread that touches this sequence's state: read above, written here
    for (int i = 0; i < hist; ++i) {
      const int t = p.S - hist + i;
      float v[8];
      if (t >= 0) {
        Vec8<__nv_bfloat16>::load(x + (long long)t * p.ldx, v);
      } else {                            // fewer new rows than the state holds: the old state moves up
        const int from = i + p.S - hist + 3;
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = from == 0 ? win[0][e] : (from == 1 ? win[1][e] : win[2][e]);
      }
      Vec8<float>::store(st + (long long)i * p.C, v);
    }
  }
  const int bw = p.C / p.blocks;
  __nv_bfloat16* o = static_cast<__nv_bfloat16*>(p.u) + (long long)(c / bw) * 2 * bw + c % bw;
  const int t1 = min(p.S, t0 + kConvRun);
#pragma unroll
  for (int i = 0; i < kConvRun; ++i) {
    const int t = t0 + i;
    if (t < t1) {
      Vec8<__nv_bfloat16>::load(x + (long long)t * p.ldx, win[(i + 3) & 3]);
      float hi[8], lo[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float acc = bias[e];
#pragma unroll
        for (int k = 0; k < 4; ++k) acc = fmaf(w[k][e], win[(i + k) & 3][e], acc);
        hi[e] = __bfloat162float(__float2bfloat16(acc));
        lo[e] = acc - hi[e];
      }
      __nv_bfloat16* dst = o + ((long long)b * p.S + t) * 2 * p.C;
      Vec8<__nv_bfloat16>::store(dst, hi);
      Vec8<__nv_bfloat16>::store(dst + bw, lo);
    }
  }
}

struct LruParams {
  const void* u;            // as written by conv_state_kernel
  float* z;                 // [B*S, blocks, 2, C / blocks] gate products without bias: recurrence gate, input gate (pass 1
                            // overwrites them)
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

// The math of one token.  The fp32 path calls the accurate functions; the bf16 path's inputs and outputs are rounded to
// 8 bits, so the hardware exponential (relative error about 2^-21) is far below them.
template <bool FAST>
__device__ __forceinline__ float exp_f(float v) { return FAST ? __expf(v) : expf(v); }
template <bool FAST>
__device__ __forceinline__ float sigmoid_f(float v) {
  return FAST ? __fdividef(1.0f, 1.0f + __expf(-v)) : 1.0f / (1.0f + expf(-v));
}
// e^v - 1 for v <= 0 with its relative precision next to 0: the Taylor polynomial of degree 7 up to 1/4
template <bool FAST>
__device__ __forceinline__ float expm1_neg_f(float v) {
  if (!FAST) return expm1f(v);
  const float t = v * fmaf(v, fmaf(v, fmaf(v, fmaf(v, fmaf(v, fmaf(v, 1.0f / 5040, 1.0f / 720), 1.0f / 120), 1.0f / 24),
                                         1.0f / 6), 0.5f), 1.0f);
  return v > -0.25f ? t : __expf(v) - 1.0f;
}
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
template <bool FAST>
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  // 1/2 (1 + tanh u) = sigmoid(2 u)
  return FAST ? z * sigmoid_f<true>(2.0f * u) : 0.5f * z * (1.0f + tanhf(u));
}

// V neighbouring channels of one sequence.
template <typename T, int V>
struct LruChannel {
  static constexpr bool FAST = sizeof(T) == 2;
  const T* u;
  float* z;
  float br[V], bi[V], decay[V];      // decay = -c * softplus(lam)
  int bw, C;
  __device__ __forceinline__ LruChannel(const LruParams& p, int b, int ch) {
    bw = p.C / p.blocks;
    C = p.C;
    const long long off = (long long)(ch / bw) * 2 * bw + ch % bw;
    const long long row0 = (long long)b * p.S;
    z = p.z + row0 * 2 * C + off;
    u = static_cast<const T*>(p.u) + (FAST ? row0 * 2 * C + off : row0 * C + ch);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      br[k] = to_f32(static_cast<const T*>(p.br)[ch + k]);
      bi[k] = to_f32(static_cast<const T*>(p.bi)[ch + k]);
      decay[k] = -p.c * softplus_f(to_f32(static_cast<const T*>(p.lam)[ch + k]));
    }
  }
  template <typename U>
  static __device__ __forceinline__ void load(const U* q, float (&o)[V]) {
    if constexpr (V == 2 && sizeof(U) == 2) {
      const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(q));
      o[0] = f.x; o[1] = f.y;
    } else if constexpr (V == 2) {
      const float2 f = *reinterpret_cast<const float2*>(q);
      o[0] = f.x; o[1] = f.y;
    } else {
      o[0] = to_f32(q[0]);
    }
  }
  static __device__ __forceinline__ void store_f32(float* q, const float (&v)[V]) {
    if constexpr (V == 2) *reinterpret_cast<float2*>(q) = make_float2(v[0], v[1]);
    else q[0] = v[0];
  }
  // What token t brings; kept apart from the arithmetic so that several tokens' loads are in flight before any store.
  struct In {
    float zr[V], zi[V], u[V];
  };
  __device__ __forceinline__ void fetch(int t, In& in) const {
    const float* zt = z + (long long)t * 2 * C;
    load(zt, in.zr);
    load(zt + bw, in.zi);
    if constexpr (FAST) {
      const T* ut = u + (long long)t * 2 * C;
      float lo[V];
      load(ut, in.u);
      load(ut + bw, lo);
#pragma unroll
      for (int k = 0; k < V; ++k) in.u[k] += lo[k];
    } else {
      load(u + (long long)t * C, in.u);
    }
  }
  // Applies a token to S; its log decay comes back in log_a.  With e = a - 1 = expm1(log a), which keeps its relative
  // precision where a is next to 1:  1 - a^2 = -e (2 + e)  and  a S = S + e S, so long memories do not drift.
  __device__ __forceinline__ void step(const In& in, float (&S)[V], float (&log_a)[V]) const {
#pragma unroll
    for (int k = 0; k < V; ++k) {
      log_a[k] = decay[k] * sigmoid_f<FAST>(in.zr[k] + br[k]);
      const float e = expm1_neg_f<FAST>(log_a[k]);
      S[k] += fmaf(e, S[k], sqrtf(-e * (2.0f + e)) * sigmoid_f<FAST>(in.zi[k] + bi[k]) * in.u[k]);
    }
  }
};

constexpr int kLruBatch = 4;      // tokens fetched at a time

template <typename T, int V>
__device__ __forceinline__ void lru_put(T* out, const float (&S)[V], const float (&y)[V]) {
  float o[V];
#pragma unroll
  for (int k = 0; k < V; ++k) o[k] = S[k] * gelu_tanh_f<sizeof(T) == 2>(y[k]);
  if constexpr (V == 2 && sizeof(T) == 2) {
    *reinterpret_cast<uint32_t*>(out) = pack_bf16x2(o[0], o[1]);
  } else {
#pragma unroll
    for (int k = 0; k < V; ++k) out[k] = from_f32<T>(o[k]);
  }
}

// The whole recurrence in one pass (chunks == 1).
template <typename T, int V>
__global__ void __launch_bounds__(128) lru_scan_kernel(const LruParams p) {
  const int ch = (blockIdx.x * 128 + threadIdx.x) * V, b = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  if (ch >= p.C) return;
  const LruChannel<T, V> lc(p, b, ch);
  float* state = p.state + (long long)b * p.C + ch;
  float S[V], la[V], y[kLruBatch][V];
  LruChannel<T, V>::load(state, S);
  const T* yp = static_cast<const T*>(p.y) + (long long)b * p.S * p.ldy + ch;
  T* out = static_cast<T*>(p.out) + (long long)b * p.S * p.C + ch;
  typename LruChannel<T, V>::In in[kLruBatch];
  for (int t0 = 0; t0 < p.S; t0 += kLruBatch) {
#pragma unroll
    for (int i = 0; i < kLruBatch; ++i) {
      if (t0 + i < p.S) {
        lc.fetch(t0 + i, in[i]);
        LruChannel<T, V>::load(yp + (long long)(t0 + i) * p.ldy, y[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < kLruBatch; ++i) {
      if (t0 + i < p.S) {
        lc.step(in[i], S, la);
        lru_put<T, V>(out + (long long)(t0 + i) * p.C, S, y[i]);
      }
    }
  }
  LruChannel<T, V>::store_f32(state, S);
}

// Pass 1.
template <typename T, int V>
__global__ void __launch_bounds__(128) lru_chunk_kernel(const LruParams p) {
  const int ch = (blockIdx.x * 128 + threadIdx.x) * V, k = blockIdx.y, b = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  if (ch >= p.C) return;
  const LruChannel<T, V> lc(p, b, ch);
  float* agg = p.agg + (long long)b * (p.chunks + 1) * 2 * p.C + ch;
  float S[V], total[V], la[V];
#pragma unroll
  for (int e = 0; e < V; ++e) S[e] = total[e] = 0.0f;
  if (k == 0) {                 // pass 2's threads of one channel start from a copy: one of them replaces the state
    float s0[V];
    LruChannel<T, V>::load(p.state + (long long)b * p.C + ch, s0);
    LruChannel<T, V>::store_f32(agg + (long long)p.chunks * 2 * p.C, s0);
  }
  const int t0 = k * p.chunk, t1 = min(p.S, t0 + p.chunk);
  typename LruChannel<T, V>::In in[kLruBatch];
  for (int t = t0; t < t1; t += kLruBatch) {
#pragma unroll
    for (int i = 0; i < kLruBatch; ++i)
      if (t + i < t1) lc.fetch(t + i, in[i]);
#pragma unroll
    for (int i = 0; i < kLruBatch; ++i) {
      if (t + i < t1) {
        lc.step(in[i], S, la);
#pragma unroll
        for (int e = 0; e < V; ++e) total[e] += la[e];
        float* zt = lc.z + (long long)(t + i) * 2 * p.C;
        LruChannel<T, V>::store_f32(zt, total);
        LruChannel<T, V>::store_f32(zt + lc.bw, S);
      }
    }
  }
  LruChannel<T, V>::store_f32(agg + (long long)k * 2 * p.C, total);
  LruChannel<T, V>::store_f32(agg + ((long long)k * 2 + 1) * p.C, S);
}

// Pass 2.
template <typename T, int V>
__global__ void __launch_bounds__(128) lru_apply_kernel(const LruParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  using Ch = LruChannel<T, V>;
  const int ch = (blockIdx.x * 128 + threadIdx.x) * V, k = blockIdx.y, b = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  if (ch >= p.C) return;
  const int bw = p.C / p.blocks;
  const float* agg = p.agg + (long long)b * (p.chunks + 1) * 2 * p.C + ch;
  float S0[V];
  Ch::load(agg + (long long)p.chunks * 2 * p.C, S0);
#pragma unroll 8
  for (int j = 0; j < k; ++j) {
    float total[V], end[V];
    Ch::load(agg + (long long)j * 2 * p.C, total);
    Ch::load(agg + ((long long)j * 2 + 1) * p.C, end);
#pragma unroll
    for (int e = 0; e < V; ++e) S0[e] += fmaf(expm1_neg_f<FAST>(total[e]), S0[e], end[e]);
  }
  const long long row0 = (long long)b * p.S;
  const float* z = p.z + row0 * 2 * p.C + (long long)(ch / bw) * 2 * bw + ch % bw;
  const T* yp = static_cast<const T*>(p.y) + row0 * p.ldy + ch;
  T* out = static_cast<T*>(p.out) + row0 * p.C + ch;
  const int t0 = k * p.chunk, t1 = min(p.S, t0 + p.chunk);
  float S[V];
  for (int t = t0; t < t1; t += kLruBatch) {
    float total[kLruBatch][V], local[kLruBatch][V], y[kLruBatch][V];
#pragma unroll
    for (int i = 0; i < kLruBatch; ++i) {
      if (t + i < t1) {
        Ch::load(z + (long long)(t + i) * 2 * p.C, total[i]);
        Ch::load(z + (long long)(t + i) * 2 * p.C + bw, local[i]);
        Ch::load(yp + (long long)(t + i) * p.ldy, y[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < kLruBatch; ++i) {
      if (t + i < t1) {
#pragma unroll
        for (int e = 0; e < V; ++e) S[e] = fmaf(exp_f<FAST>(total[i][e]), S0[e], local[i][e]);
        lru_put<T, V>(out + (long long)(t + i) * p.C, S, y[i]);
      }
    }
  }
  if (k == p.chunks - 1) Ch::store_f32(p.state + (long long)b * p.C + ch, S);
}

template <typename T, int V>
static int launch_lru(const LruParams& p, cudaStream_t st) {
  const unsigned gx = (p.C / V + 127) / 128;
  if (p.chunks == 1) return counted(1, (int)launch_k(lru_scan_kernel<T, V>, dim3(gx, 1, p.B), dim3(128), (size_t)0, st, p));
  const dim3 grid(gx, p.chunks, p.B);
  const int rc = counted(1, (int)launch_k(lru_chunk_kernel<T, V>, grid, dim3(128), (size_t)0, st, p));
  if (rc) return rc;
  return counted(1, (int)launch_k(lru_apply_kernel<T, V>, grid, dim3(128), (size_t)0, st, p));
}

}  // namespace dptb

using namespace dptb;

struct DptbRecurrentArgs {
  const void* x; const void* taps; const void* conv_bias; float* conv_state; void* u;     // convolution
  float* z; const void* br; const void* bi; const void* lam; const void* y;         // recurrence
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
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (!a->f32 && a->K <= 4 && (a->C / a->blocks) % 8 == 0 && a->ldx % 8 == 0 && al16(a->x) && al16(a->conv_bias) && al16(a->u) &&
      (a->K == 1 || al16(a->conv_state))) {
    const long long runs = (a->S + kConvRun - 1) / kConvRun * (long long)a->B;
    const unsigned cy = (a->C / 8 + 127) / 128;
    if (runs > 0x7fffffff || cy > 65535) return kErrTooLarge;
    return counted(1, (int)launch_k(conv_state_vec_kernel, dim3((unsigned)runs, cy), dim3(128), (size_t)0, st, p));
  }
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
  if (p.chunks > 1 && (!a->agg || a->agg_floats < (long long)a->B * (p.chunks + 1) * 2 * a->C)) return kErrTooLarge;
  auto al4 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 3) == 0; };
  auto al8 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 7) == 0; };
  const bool pairs = (a->C / a->blocks) % 2 == 0 && a->ldy % 2 == 0 && al4(a->u) && al4(a->y) && al4(a->out) && al8(a->z) &&
                     al8(a->state) && al8(a->agg);
  if (a->f32) return launch_lru<float, 1>(p, st);
  // narrow inputs need the threads more than the wider accesses
  if (pairs && (long long)a->B * p.chunks * a->C >= 256 * 1024) return launch_lru<__nv_bfloat16, 2>(p, st);
  return launch_lru<__nv_bfloat16, 1>(p, st);
}
