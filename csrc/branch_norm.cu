// The residual stream (fp32) of a decoder that normalises what a sublayer returns, and averages over depth:
//
//   x'  = x + rms(c_1 m_1 + c_2 m_2) * w            a sublayer's result; m_2 optional; x may be an embedding row
//   x'' = sum_{j < n} a_j X_j + a_n x'              optional: X_j are results of earlier layers (a stack of streams)
//   h   = x'' in the sublayers' dtype               or  rms(x'') * w_f, the norm in front of the output
//
// One kernel between two sublayers: a CTA per row, everything of a row in registers.
#include <cuda_bf16.h>

#include <type_traits>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

struct BranchParams {
  const float* x;             // [rows, D] or null (then the embedding row is the stream)
  const void* embed;          // [vocab, D]
  const long long* tokens;    // [rows]
  const void* m1;             // [rows, D] or null (nothing is added)
  const void* m2;
  const void* w;              // [D]
  const float* stack;         // [n, rows of the step, D] earlier results; null: no average
  const void* avg;            // [n + 1] weights
  const int* pick;            // output row r is source row pick[r]
  const void* wf;             // [D]: h = rms(x'') * wf
  float* result;              // [rows, D] x'
  float* x_out;               // [rows, D] x''
  void* h;                    // [rows, D] or null
  long long stack_stride;
  int rows, D, n, vocab;
  float c1, c2, eps;
};

constexpr int kBranchThreads = 256;   // at most

template <typename T, int V, int NV>
__global__ void __launch_bounds__(kBranchThreads) branch_norm_kernel(const BranchParams p) {
  __shared__ float scratch[33];
  pdl_wait();
  pdl_launch_dependents();
  const long long out = blockIdx.x, r = p.pick ? p.pick[out] : out;
  auto col = [](int i) { return (i * (int)blockDim.x + (int)threadIdx.x) * V; };
  auto load = [](const auto* q, float (&o)[V]) {
    using U = std::remove_cv_t<std::remove_pointer_t<decltype(q)>>;
    if constexpr (V == 8) Vec8<U>::load(q, o);
    else o[0] = to_f32(q[0]);
  };
  auto store = [](auto* q, const float (&o)[V]) {
    using U = std::remove_pointer_t<decltype(q)>;
    if constexpr (V == 8) Vec8<U>::store(q, o);
    else q[0] = from_f32<U>(o[0]);
  };
  float x[NV][V], m[NV][V];
  const long long tok = p.embed ? p.tokens[r] : 0;
  const bool emb = p.embed && tok >= 0 && tok < p.vocab;
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = col(i);
#pragma unroll
    for (int k = 0; k < V; ++k) x[i][k] = m[i][k] = 0.0f;
    if (c >= p.D) continue;
    if (p.x) load(p.x + r * p.D + c, x[i]);
    else if (emb) load(static_cast<const T*>(p.embed) + tok * p.D + c, x[i]);
    if (p.m1) {
      load(static_cast<const T*>(p.m1) + r * p.D + c, m[i]);
#pragma unroll
      for (int k = 0; k < V; ++k) m[i][k] *= p.c1;
      if (p.m2) {
        float t[V];
        load(static_cast<const T*>(p.m2) + r * p.D + c, t);
#pragma unroll
        for (int k = 0; k < V; ++k) m[i][k] = fmaf(p.c2, t[k], m[i][k]);
      }
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(m[i][k], m[i][k], ss);
    }
  }
  if (p.m1) {
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.D + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (col(i) >= p.D) continue;
      float w[V];
      load(static_cast<const T*>(p.w) + col(i), w);
#pragma unroll
      for (int k = 0; k < V; ++k) x[i][k] = fmaf(m[i][k] * inv, w[k], x[i][k]);
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (p.result && col(i) < p.D) store(p.result + out * p.D + col(i), x[i]);
  if (p.stack) {
    const T* a = static_cast<const T*>(p.avg);
    const float own = to_f32(a[p.n]);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = col(i);
      if (c >= p.D) continue;
#pragma unroll
      for (int k = 0; k < V; ++k) m[i][k] = 0.0f;
      const float* s = p.stack + r * p.D + c;
#pragma unroll 4
      for (int j = 0; j < p.n; ++j) {
        float t[V];
        load(s + j * p.stack_stride, t);
        const float aj = to_f32(a[j]);
#pragma unroll
        for (int k = 0; k < V; ++k) m[i][k] = fmaf(aj, t[k], m[i][k]);
      }
#pragma unroll
      for (int k = 0; k < V; ++k) x[i][k] = fmaf(own, x[i][k], m[i][k]);
    }
  }
  float inv = 1.0f;
  if (p.wf) {
    ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(x[i][k], x[i][k], ss);
    inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.D + p.eps);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = col(i);
    if (c >= p.D) continue;
    if (p.x_out) store(p.x_out + out * p.D + c, x[i]);
    if (p.h) {
      float y[V];
      if (p.wf) load(static_cast<const T*>(p.wf) + c, y);
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] = p.wf ? x[i][k] * inv * y[k] : x[i][k];
      store(static_cast<T*>(p.h) + out * p.D + c, y);
    }
  }
}

template <typename T, int V, int NV>
static int launch_branch(const BranchParams& p, cudaStream_t st) {
  const int threads = (((p.D + V * NV - 1) / (V * NV)) + 31) / 32 * 32;
  return counted(1, (int)launch_k(branch_norm_kernel<T, V, NV>, dim3((unsigned)p.rows), dim3(threads), (size_t)0, st, p));
}
template <typename T>
static int dispatch_branch(const BranchParams& p, bool vec, cudaStream_t st) {
  const int nv = (p.D + (vec ? 8 : 1) * kBranchThreads - 1) / ((vec ? 8 : 1) * kBranchThreads);
  if (vec) {
    if (nv <= 1) return launch_branch<T, 8, 1>(p, st);
    if (nv <= 2) return launch_branch<T, 8, 2>(p, st);
    if (nv <= 4) return launch_branch<T, 8, 4>(p, st);
    return kErrUnsupported;
  }
  if (nv <= 2) return launch_branch<T, 1, 2>(p, st);
  if (nv <= 8) return launch_branch<T, 1, 8>(p, st);
  if (nv <= 32) return launch_branch<T, 1, 32>(p, st);
  return kErrUnsupported;
}

}  // namespace dptb

using namespace dptb;

struct DptbBranchArgs {
  const float* x; const void* embed; const long long* tokens; const void* m1; const void* m2; const void* w;
  const float* stack; const void* avg; const int* pick; const void* wf; float* result; float* x_out; void* h;
  long long stack_stride;
  int rows, D, n, vocab, f32;
  float c1, c2, eps;
};

extern "C" int dptb_branch_norm(const DptbBranchArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->rows <= 0) return 0;
  if (a->D <= 0 || (!a->x && (!a->embed || !a->tokens)) || (a->m1 && !a->w) || (a->m2 && !a->m1)) return kErrBadShape;
  if (a->stack && (!a->avg || a->n < 0)) return kErrBadShape;
  if (a->pick && (a->x_out == a->x && a->x_out)) return kErrBadShape;
  BranchParams p;
  p.x = a->x; p.embed = a->embed; p.tokens = a->tokens; p.m1 = a->m1; p.m2 = a->m2; p.w = a->w;
  p.stack = a->stack; p.avg = a->avg; p.pick = a->pick; p.wf = a->wf; p.result = a->result; p.x_out = a->x_out; p.h = a->h;
  p.stack_stride = a->stack_stride; p.rows = a->rows; p.D = a->D; p.n = a->n; p.vocab = a->vocab;
  p.c1 = a->c1; p.c2 = a->c2; p.eps = a->eps;
  bool vec = a->D % 8 == 0 && a->stack_stride % 8 == 0;
  for (const void* q : {(const void*)a->x, a->embed, a->m1, a->m2, a->w, (const void*)a->stack, a->wf,
                        (const void*)a->result, (const void*)a->x_out, (const void*)a->h})
    vec = vec && (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  return a->f32 ? dispatch_branch<float>(p, vec, st) : dispatch_branch<__nv_bfloat16>(p, vec, st);
}
