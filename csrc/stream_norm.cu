// The residual stream of a decoder whose residual is kept in fp32: one kernel between two layers.
//
//   x'  = x + (mix + shared + sum_k w_k y[slot_k])  (+ embed[token])        every term optional; x may be an embedding row
//   n1  = x' / sqrt(mean(x'^2) + eps) * g1,   n2 = the same with g2         (g: one number)
//   h1_t = n1_t + (n1_{t-1} - n1_t) * shift                                 previous token's n1 from the state at a
//                                                                           sequence's first row; h1 = n1 without a shift
// It closes a layer (both branches' outputs, the experts' weighted sum) and opens the next one (both norms, the token
// shift), so the stream is read and written once per layer.  A CTA walks a run of consecutive rows and keeps the previous
// row's n1 in registers; the row before the run is recomputed.  x is never updated in place (a neighbour recomputes rows).
// The CTA of a sequence's first row reads the shift state and afterwards writes the new one, so that no other CTA can
// overwrite what it still reads.
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

struct StreamParams {
  const float* x;             // [rows, D] or null (then the embedding row is the stream)
  const void* mix;            // [rows, D]
  const void* shared;         // [rows, D]
  const void* y;              // [*, D] expert outputs
  const int* slot;            // [rows, top]
  const float* w;             // [rows, top]
  const void* embed;          // [vocab, D]
  const long long* tokens;    // [rows]
  const int* pick;            // output row r is source row pick[r] (no shift then)
  const void* g1;
  const void* g2;
  const void* shift;          // [D]
  float* shift_state;         // [B, D]
  float* x_out;
  void* h1;
  void* h2;
  int rows, S, D, top, vocab, run;
  float eps;
};

constexpr int kStreamThreads = 256;   // at most

// V consecutive columns per load, NV loads per thread.
template <typename T, int V, int NV>
struct StreamRow {
  float v[NV][V];
  static __device__ __forceinline__ int col(int i) { return (i * blockDim.x + threadIdx.x) * V; }
  template <typename U>
  static __device__ __forceinline__ void load(const U* p, float (&o)[V]) {
    if constexpr (V == 8) Vec8<U>::load(p, o);
    else o[0] = to_f32(p[0]);
  }
  template <typename U>
  static __device__ __forceinline__ void store(U* p, const float (&o)[V]) {
    if constexpr (V == 8) Vec8<U>::store(p, o);
    else p[0] = from_f32<U>(o[0]);
  }
  // the stream after this layer, row r
  __device__ __forceinline__ void compute(const StreamParams& p, long long r) {
    const long long tok = p.tokens ? p.tokens[r] : 0;
    const bool emb = p.embed && tok >= 0 && tok < p.vocab;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = col(i);
      float d[V];
#pragma unroll
      for (int k = 0; k < V; ++k) v[i][k] = d[k] = 0.0f;
      if (c >= p.D) continue;
      float t[V];
      if (p.x) load(p.x + r * p.D + c, v[i]);
      if (p.mix) load(static_cast<const T*>(p.mix) + r * p.D + c, d);
      if (p.shared) {
        load(static_cast<const T*>(p.shared) + r * p.D + c, t);
#pragma unroll
        for (int k = 0; k < V; ++k) d[k] += t[k];
      }
      for (int j0 = 0; j0 < p.top; j0 += 4) {      // four experts' rows in flight
        float yt[4][V], w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const bool on = j0 + j < p.top;
          const long long at = r * p.top + (on ? j0 + j : 0);
          w[j] = on ? p.w[at] : 0.0f;
          load(static_cast<const T*>(p.y) + (long long)p.slot[at] * p.D + c, yt[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int k = 0; k < V; ++k) d[k] = j0 + j < p.top ? fmaf(w[j], yt[j][k], d[k]) : d[k];
      }
#pragma unroll
      for (int k = 0; k < V; ++k) v[i][k] += d[k];
      if (emb) {
        load(static_cast<const T*>(p.embed) + tok * p.D + c, t);
#pragma unroll
        for (int k = 0; k < V; ++k) v[i][k] += t[k];
      }
    }
  }
  __device__ __forceinline__ float inv_rms(const StreamParams& p, float* scratch) const {
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(v[i][k], v[i][k], ss);
    return 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.D + p.eps);
  }
};

template <typename T, int V, int NV>
__global__ void __launch_bounds__(kStreamThreads) stream_norm_kernel(const StreamParams p) {
  using Row = StreamRow<T, V, NV>;
  __shared__ float scratch[33];
  pdl_wait();
  pdl_launch_dependents();
  const float g1 = to_f32(*static_cast<const T*>(p.g1));
  const float g2 = p.g2 ? to_f32(*static_cast<const T*>(p.g2)) : 0.0f;
  const long long r0 = (long long)blockIdx.x * p.run;
  const long long r1 = min((long long)p.rows, r0 + p.run);
  Row cur;
  float prev[NV][V];
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int k = 0; k < V; ++k) prev[i][k] = 0.0f;

  if (p.shift && r0 % p.S != 0) {     // the row before the run
    cur.compute(p, r0 - 1);
    const float s = cur.inv_rms(p, scratch) * g1;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int k = 0; k < V; ++k) prev[i][k] = cur.v[i][k] * s;
  }
  for (long long r = r0; r < r1; ++r) {
    if (p.shift && r % p.S == 0) {
      float* state = p.shift_state + (r / p.S) * p.D;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (Row::col(i) < p.D) Row::load(state + Row::col(i), prev[i]);
      if (p.S > 1) {
        cur.compute(p, r + p.S - 1);    // the sequence's last row becomes the state
        const float s = cur.inv_rms(p, scratch) * g1;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          float n[V];
#pragma unroll
          for (int k = 0; k < V; ++k) n[k] = cur.v[i][k] * s;
          if (Row::col(i) < p.D) Row::store(state + Row::col(i), n);
        }
      }
    }
    cur.compute(p, p.pick ? (long long)p.pick[r] : r);
    const float inv = cur.inv_rms(p, scratch);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = Row::col(i);
      float n[V], h[V];
#pragma unroll
      for (int k = 0; k < V; ++k) n[k] = cur.v[i][k] * inv * g1;
      if (c < p.D) {
        if (p.x_out) Row::store(p.x_out + r * p.D + c, cur.v[i]);
        if (p.shift) {
          float mu[V];
          Row::load(static_cast<const T*>(p.shift) + c, mu);
#pragma unroll
          for (int k = 0; k < V; ++k) h[k] = fmaf(prev[i][k] - n[k], mu[k], n[k]);
          if (p.S == 1) Row::store(p.shift_state + r * p.D + c, n);
          Row::store(static_cast<T*>(p.h1) + r * p.D + c, h);
        } else {
          Row::store(static_cast<T*>(p.h1) + r * p.D + c, n);
        }
        if (p.h2) {
#pragma unroll
          for (int k = 0; k < V; ++k) h[k] = cur.v[i][k] * inv * g2;
          Row::store(static_cast<T*>(p.h2) + r * p.D + c, h);
        }
      }
#pragma unroll
      for (int k = 0; k < V; ++k) prev[i][k] = n[k];
    }
  }
}

template <typename T, int V, int NV>
static int launch_stream(const StreamParams& p, cudaStream_t st) {
  const dim3 grid((unsigned)((p.rows + p.run - 1) / p.run));
  const int threads = (((p.D + V * NV - 1) / (V * NV)) + 31) / 32 * 32;
  return counted(1, (int)launch_k(stream_norm_kernel<T, V, NV>, grid, dim3(threads), (size_t)0, st, p));
}
template <typename T>
static int dispatch_stream(const StreamParams& p, bool vec, cudaStream_t st) {
  if (vec) {
    const int nv = (p.D + 8 * kStreamThreads - 1) / (8 * kStreamThreads);
    if (nv <= 1) return launch_stream<T, 8, 1>(p, st);
    if (nv <= 2) return launch_stream<T, 8, 2>(p, st);
    if (nv <= 4) return launch_stream<T, 8, 4>(p, st);
    return kErrUnsupported;
  }
  const int nv = (p.D + kStreamThreads - 1) / kStreamThreads;
  if (nv <= 2) return launch_stream<T, 1, 2>(p, st);
  if (nv <= 8) return launch_stream<T, 1, 8>(p, st);
  if (nv <= 32) return launch_stream<T, 1, 32>(p, st);
  return kErrUnsupported;
}

}  // namespace dptb

using namespace dptb;

struct DptbStreamArgs {
  const float* x; const void* mix; const void* shared; const void* y; const int* slot; const float* w;
  const void* embed; const long long* tokens; const int* pick; const void* g1; const void* g2; const void* shift;
  float* shift_state; float* x_out; void* h1; void* h2;
  int rows, S, D, top, vocab, f32;
  float eps;
};

extern "C" int dptb_stream_norm(const DptbStreamArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->rows <= 0) return 0;
  if (a->D <= 0 || a->S <= 0 || !a->h1 || !a->g1 || (!a->x && !a->embed) || (a->embed && !a->tokens)) return kErrBadShape;
  if (a->shift && (!a->shift_state || a->pick || a->rows % a->S)) return kErrBadShape;
  if (a->top > 0 && (!a->y || !a->slot || !a->w)) return kErrBadShape;
  if (a->x_out && a->x_out == a->x) return kErrBadShape;
  StreamParams p;
  p.x = a->x; p.mix = a->mix; p.shared = a->shared; p.y = a->y; p.slot = a->slot; p.w = a->w;
  p.embed = a->embed; p.tokens = a->tokens; p.pick = a->pick; p.g1 = a->g1; p.g2 = a->g2; p.shift = a->shift;
  p.shift_state = a->shift_state; p.x_out = a->x_out; p.h1 = a->h1; p.h2 = a->h2;
  p.rows = a->rows; p.S = a->S; p.D = a->D; p.top = a->top > 0 ? a->top : 0; p.vocab = a->vocab; p.eps = a->eps;
  // runs of up to 8 rows, as long as two CTAs per SM remain (without a shift rows are independent)
  p.run = 1;
  while (a->shift && p.run < 8 && a->rows / (2 * p.run) >= 2 * sm_count()) p.run *= 2;
  bool vec = a->D % 8 == 0;
  for (const void* q : {(const void*)a->x, a->mix, a->shared, a->y, a->embed, a->shift, (const void*)a->shift_state,
                        (const void*)a->x_out, (const void*)a->h1, (const void*)a->h2})
    vec = vec && (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  return a->f32 ? dispatch_stream<float>(p, vec, st) : dispatch_stream<__nv_bfloat16>(p, vec, st);
}
