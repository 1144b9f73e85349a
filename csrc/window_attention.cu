// Windowed attention around the two attention kernels: what happens to a projected row before it is a query, key or value,
// the cache of the window, the pooled blocks before it, and a generic attention kernel.
//
// Cache of a sequence: a ring of `ring` token rows (the row of position p is p % ring) and one row for every block of `pool`
// tokens, the mean of the block's keys (values) as the ring holds them.  The query at position i sees the positions
// i - window < j <= i and, with pooling, the blocks b with (b + 1) * pool <= i - window + 1.  The ring is longer than the
// window by the longest step that reads it in place; longer steps work on a linear copy ([history | new tokens]).
//
//   qkv_prep       norm of q and k (per head, or over all heads together), rotation by position, values turned by position,
//                  rows into the ring (and the linear copy)
//   pool_blocks    means of the blocks that are complete
//   window_attn    any dtype and size: a CTA per (query, head); steps of bf16 use the flash and decode kernels instead
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

struct PrepParams {
  const void* p;            // [B*S, ld] projected rows
  long long ld;
  int oq, ok, ov;           // columns of q, k, v
  const void* gq;           // norm weights, [H * dk] / [G * dk] (whole) or [dk]; null: no norm
  const void* gk;
  const float2* rot;        // [positions, rot_dims / 2] (cos, sin)
  const float2* rot_v;      // [positions, dv / 2] or null
  void* q;                  // [B*S, H * dk]
  void* k_ring;             // [B, ring, G * dk]
  void* v_ring;             // [B, ring, G * dv]
  void* k_lin;              // [B, lin_rows, G * dk] or null; token s goes to row hist + s
  void* v_lin;
  void* k_pool;             // [B, pool_rows, G * dk] or null: the block that ended just before this step (S == 1)
  void* v_pool;
  const int* pos_ptr;
  int B, S, H, G, dk, dv, whole, rot_dims, ring, lin_rows, hist, pos, rot_rows, pool, pool_rows;
  float eps;
};

constexpr int kPrepThreads = 256;

// The mean of the block of `pool` rows that starts at position p0, features c ... c + V - 1.
template <typename T, int V>
__device__ __forceinline__ void block_mean(const T* rows, long long ld, int c, int p0, int pool, int ring, int lin0, T* out) {
  float s[V];
#pragma unroll
  for (int e = 0; e < V; ++e) s[e] = 0.0f;
  const int start = ring ? p0 % ring : p0 - lin0;
#pragma unroll 8
  for (int j = 0; j < pool; ++j) {
    const int at = ring && start + j >= ring ? start + j - ring : start + j;
    const T* r = rows + at * ld + c;
    float v[V];
    if constexpr (V == 8) Vec8<T>::load(r, v);
    else v[0] = to_f32(r[0]);
#pragma unroll
    for (int e = 0; e < V; ++e) s[e] += v[e];
  }
#pragma unroll
  for (int e = 0; e < V; ++e) s[e] /= (float)pool;
  if constexpr (V == 8) Vec8<T>::store(out, s);
  else out[0] = from_f32<T>(s[0]);
}

// One CTA per token.  Rows are staged in shared memory as fp32; V consecutive features per thread and access.
template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) qkv_prep_kernel(const PrepParams p) {
  extern __shared__ float prep_smem[];        // q and k features, then one factor per head
  __shared__ float scratch[33];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = blockIdx.x, b = row / p.S, s = row % p.S;
  const int nq = p.H * p.dk, nk = p.G * p.dk, nv = p.G * p.dv;
  float* x = prep_smem;
  float* inv = prep_smem + nq + nk;           // [H + G]
  pdl_wait();
  pdl_launch_dependents();
  const int pos0 = p.pos_ptr ? *p.pos_ptr : p.pos, pos = pos0 + s;
  if (pos < 0 || pos >= p.rot_rows) {
    if (tid == 0) report_error(kBadArgument);
    return;
  }
  auto load = [&](const T* q, float (&o)[V]) {
    if constexpr (V == 8) Vec8<T>::load(q, o);
    else o[0] = to_f32(q[0]);
  };
  auto store = [&](T* q, const float (&o)[V]) {
    if constexpr (V == 8) Vec8<T>::store(q, o);
    else q[0] = from_f32<T>(o[0]);
  };
  const T* src = static_cast<const T*>(p.p) + (long long)row * p.ld;
  float sq = 0.0f, sk = 0.0f;
  for (int c = tid * V; c < nq + nk; c += kPrepThreads * V) {
    float v[V];
    load(c < nq ? src + p.oq + c : src + p.ok + c - nq, v);
    if constexpr (V == 8) Vec8<float>::store(x + c, v);
    else x[c] = v[0];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      if (c < nq) sq = fmaf(v[e], v[e], sq);
      else sk = fmaf(v[e], v[e], sk);
    }
  }
  if (p.gq) {
    if (p.whole) {
      sq = block_sum(sq, scratch);
      sk = block_sum(sk, scratch);
      const float iq = 1.0f / sqrtf(sq / (float)nq + p.eps), ik = 1.0f / sqrtf(sk / (float)nk + p.eps);
      for (int h = tid; h < p.H + p.G; h += kPrepThreads) inv[h] = h < p.H ? iq : ik;
    } else {
      __syncthreads();
      for (int h = warp; h < p.H + p.G; h += kPrepThreads / 32) {
        float ss = 0.0f;
        for (int c = lane; c < p.dk; c += 32) ss = fmaf(x[h * p.dk + c], x[h * p.dk + c], ss);
        ss = warp_sum(ss);
        if (lane == 0) inv[h] = 1.0f / sqrtf(ss / (float)p.dk + p.eps);
      }
    }
  }
  __syncthreads();
  T* k_ring = static_cast<T*>(p.k_ring) + ((long long)b * p.ring + pos % p.ring) * nk;
  T* v_ring = static_cast<T*>(p.v_ring) + ((long long)b * p.ring + pos % p.ring) * nv;
  const bool keep = s >= p.S - p.ring;        // an earlier token's row would be overwritten by this step's own
  const long long lin = (long long)b * p.lin_rows + p.hist + s;
  const float2* rot = p.rot + (long long)pos * (p.rot_dims / 2);
  auto normed = [&](int c, int d, float (&v)[V]) {     // features c ... of [q | k] (feature d of their head) after the norm
    if constexpr (V == 8) Vec8<float>::load(x + c, v);
    else v[0] = x[c];
    if (!p.gq) return;
    const bool is_k = c >= nq;
    float g[V];
    load(static_cast<const T*>(is_k ? p.gk : p.gq) + (p.whole ? (is_k ? c - nq : c) : d), g);
    const float s = inv[(c - d) / p.dk];
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= s * g[e];
  };
  for (int c = tid * V; c < nq + nk; c += kPrepThreads * V) {
    float v[V];
    const int d = c % p.dk;
    normed(c, d, v);
    if constexpr (V == 8) {
#pragma unroll
      for (int e = 0; e < V; e += 2) {
        if (d + e < p.rot_dims) {
          const float2 cs = rot[(d + e) / 2];
          const float a = v[e], o = v[e + 1];
          v[e] = a * cs.x - o * cs.y;
          v[e + 1] = o * cs.x + a * cs.y;
        }
      }
    } else if (d < p.rot_dims) {
      float o[V];
      const int step = d & 1 ? -1 : 1;
      normed(c + step, d + step, o);
      const float2 cs = rot[d / 2];
      v[0] = d & 1 ? v[0] * cs.x + o[0] * cs.y : v[0] * cs.x - o[0] * cs.y;
    }
    if (c < nq) {
      store(static_cast<T*>(p.q) + (long long)row * nq + c, v);
    } else {
      if (keep) store(k_ring + c - nq, v);
      if (p.k_lin) store(static_cast<T*>(p.k_lin) + lin * nk + c - nq, v);
    }
  }
  const float2* rot_v = p.rot_v ? p.rot_v + (long long)pos * (p.dv / 2) : nullptr;
  for (int c = tid * V; c < nv; c += kPrepThreads * V) {
    float v[V];
    load(src + p.ov + c, v);
    const int d = c % p.dv;
    if (rot_v) {
      if constexpr (V == 8) {
#pragma unroll
        for (int e = 0; e < V; e += 2) {
          const float2 cs = rot_v[(d + e) / 2];
          const float a = v[e], o = v[e + 1];
          v[e] = a * cs.x - o * cs.y;
          v[e + 1] = o * cs.x + a * cs.y;
        }
      } else if ((d | 1) < p.dv) {
        const float2 cs = rot_v[d / 2];
        const float o = to_f32(src[p.ov + (d & 1 ? c - 1 : c + 1)]);
        v[0] = d & 1 ? v[0] * cs.x + o * cs.y : v[0] * cs.x - o * cs.y;
      }
    }
    if (keep) store(v_ring + c, v);
    if (p.v_lin) store(static_cast<T*>(p.v_lin) + lin * nv + c, v);
  }
  // decoding: the block that the previous step completed (all of its rows are older than this step)
  if (p.k_pool && pos > 0 && pos % p.pool == 0 && pos / p.pool <= p.pool_rows) {
    const int blk = pos / p.pool - 1;
    const T* kr = static_cast<const T*>(p.k_ring) + (long long)b * p.ring * nk;
    const T* vr = static_cast<const T*>(p.v_ring) + (long long)b * p.ring * nv;
    T* kp = static_cast<T*>(p.k_pool) + ((long long)b * p.pool_rows + blk) * nk;
    T* vp = static_cast<T*>(p.v_pool) + ((long long)b * p.pool_rows + blk) * nv;
    for (int c = tid * V; c < nk; c += kPrepThreads * V) block_mean<T, V>(kr, nk, c, blk * p.pool, p.pool, p.ring, 0, kp + c);
    for (int c = tid * V; c < nv; c += kPrepThreads * V) block_mean<T, V>(vr, nv, c, blk * p.pool, p.pool, p.ring, 0, vp + c);
  }
}

struct PoolParams {
  const void* k;            // token rows: a ring (ring > 0) or linear from position lin0
  const void* v;
  long long k_batch, v_batch;   // elements between sequences
  void* k_pool;             // [B, pool_rows, nk]
  void* v_pool;
  int nk, nv, ring, lin0, pool, pool_rows, first;   // blocks first + blockIdx.x
};

constexpr int kPoolThreads = 128;

template <typename T, int V>
__global__ void __launch_bounds__(kPoolThreads) pool_blocks_kernel(const PoolParams p) {
  const int blk = p.first + blockIdx.x, b = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const T* k = static_cast<const T*>(p.k) + b * p.k_batch;
  const T* v = static_cast<const T*>(p.v) + b * p.v_batch;
  T* kp = static_cast<T*>(p.k_pool) + ((long long)b * p.pool_rows + blk) * p.nk;
  T* vp = static_cast<T*>(p.v_pool) + ((long long)b * p.pool_rows + blk) * p.nv;
  for (int c = threadIdx.x * V; c < p.nk + p.nv; c += kPoolThreads * V) {
    if (c < p.nk) block_mean<T, V>(k, p.nk, c, blk * p.pool, p.pool, p.ring, p.lin0, kp + c);
    else block_mean<T, V>(v, p.nv, c - p.nk, blk * p.pool, p.pool, p.ring, p.lin0, vp + c - p.nk);
  }
}

struct WindowParams {
  const void* q;            // [B*S, H * dk]
  const void* k;
  const void* v;
  const void* k_pool;
  const void* v_pool;
  const void* sink;         // [H] or null
  const float2* rot_v;      // outputs are turned back by their position; null: not
  void* o;                  // [B*S, H * dv]
  long long k_batch, v_batch;
  const int* pos_ptr;
  int B, S, H, G, dk, dv, ring, lin0, window, pool, pool_rows, pos;
  float scale;
};

// 4 warps per (query, head), every warp takes every fourth key with its own running softmax.  MAXV * 32 >= dk, dv.
template <typename T, int MAXV>
__global__ void __launch_bounds__(128) window_attn_kernel(const WindowParams p) {
  __shared__ float red[4][MAXV * 32 + 2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, row = blockIdx.x;
  const int b = row / p.S, g = h / (p.H / p.G);
  pdl_wait();
  pdl_launch_dependents();
  const int i = (p.pos_ptr ? *p.pos_ptr : p.pos) + row % p.S;
  const int lo = max(0, i - p.window + 1);
  const int blocks = p.pool > 0 && i - p.window + 1 >= p.pool ? min((i - p.window + 1) / p.pool, p.pool_rows) : 0;
  const int n = blocks + i - lo + 1;
  const int nk = p.G * p.dk, nv = p.G * p.dv;
  const T* q = static_cast<const T*>(p.q) + ((long long)row * p.H + h) * p.dk;
  const T* kt = static_cast<const T*>(p.k) + b * p.k_batch + g * p.dk;
  const T* vt = static_cast<const T*>(p.v) + b * p.v_batch + g * p.dv;
  const T* kp = static_cast<const T*>(p.k_pool) + (long long)b * p.pool_rows * nk + g * p.dk;
  const T* vp = static_cast<const T*>(p.v_pool) + (long long)b * p.pool_rows * nv + g * p.dv;
  float qv[MAXV], o[MAXV];
#pragma unroll
  for (int e = 0; e < MAXV; ++e) {
    const int c = e * 32 + lane;
    qv[e] = c < p.dk ? to_f32(q[c]) : 0.0f;
    o[e] = 0.0f;
  }
  // the sink takes part in the sum of one warp: a score without a key
  float m = -INFINITY, l = 0.0f;
  if (p.sink && warp == 0) {
    m = to_f32(static_cast<const T*>(p.sink)[h]);
    l = 1.0f;
  }
  for (int j = warp; j < n; j += 4) {
    const T *k, *v;
    if (j < blocks) {
      k = kp + (long long)j * nk;
      v = vp + (long long)j * nv;
    } else {
      const int at = lo + j - blocks;
      const long long r = p.ring ? at % p.ring : at - p.lin0;
      k = kt + r * nk;
      v = vt + r * nv;
    }
    float s = 0.0f, vv[MAXV];
#pragma unroll
    for (int e = 0; e < MAXV; ++e) {
      const int c = e * 32 + lane;
      if (c < p.dk) s = fmaf(qv[e], to_f32(k[c]), s);
      vv[e] = c < p.dv ? to_f32(v[c]) : 0.0f;
    }
    s = warp_sum(s) * p.scale;
    const float m_new = fmaxf(m, s);
    const float al = expf(m - m_new), w = expf(s - m_new);
    l = l * al + w;
#pragma unroll
    for (int e = 0; e < MAXV; ++e) o[e] = fmaf(w, vv[e], o[e] * al);
    m = m_new;
  }
#pragma unroll
  for (int e = 0; e < MAXV; ++e) red[warp][e * 32 + lane] = o[e];
  if (lane == 0) {
    red[warp][MAXV * 32] = m;
    red[warp][MAXV * 32 + 1] = l;
  }
  __syncthreads();
  float mm = -INFINITY, ll = 0.0f, wt[4];
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, red[w][MAXV * 32]);
  for (int w = 0; w < 4; ++w) {
    wt[w] = red[w][MAXV * 32] == -INFINITY ? 0.0f : expf(red[w][MAXV * 32] - mm);
    ll += red[w][MAXV * 32 + 1] * wt[w];
  }
  const float inv = 1.0f / ll;
  auto value = [&](int c) {
    float v = 0.0f;
    for (int w = 0; w < 4; ++w) v += red[w][c] * wt[w];
    return v * inv;
  };
  T* out = static_cast<T*>(p.o) + ((long long)row * p.H + h) * p.dv;
  for (int c = threadIdx.x; c < p.dv; c += 128) {
    float v = value(c);
    if (p.rot_v && (c | 1) < p.dv) {
      const float2 cs = p.rot_v[(long long)i * (p.dv / 2) + c / 2];
      const float u = value(c ^ 1);
      v = c & 1 ? v * cs.x - u * cs.y : v * cs.x + u * cs.y;
    }
    out[c] = from_f32<T>(v);
  }
}

template <typename T>
static int launch_window(const WindowParams& p, cudaStream_t st) {
  const dim3 grid(p.B * p.S, p.H);
  const int d = p.dk > p.dv ? p.dk : p.dv;
#define DPTB_WIN(M) return counted(1, (int)launch_k(window_attn_kernel<T, M>, grid, dim3(128), (size_t)0, st, p))
  if (d <= 64) DPTB_WIN(2);
  if (d <= 128) DPTB_WIN(4);
  if (d <= 256) DPTB_WIN(8);
  if (d <= 512) DPTB_WIN(16);
  if (d <= 1024) DPTB_WIN(32);
#undef DPTB_WIN
  return kErrUnsupported;
}

}  // namespace dptb

using namespace dptb;

struct DptbPrepArgs {
  const void* p; const void* gq; const void* gk; const void* rot; const void* rot_v; void* q; void* k_ring; void* v_ring;
  void* k_lin; void* v_lin; void* k_pool; void* v_pool; const int* pos_ptr;
  long long ld;
  int oq, ok, ov, B, S, H, G, dk, dv, whole, rot_dims, ring, lin_rows, hist, pos, rot_rows, pool, pool_rows, f32;
  float eps;
};

extern "C" int dptb_qkv_prep(const DptbPrepArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->S <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || a->H % a->G || a->dk <= 0 || a->dv <= 0 || a->ring <= 0) return kErrBadShape;
  if (a->rot_dims < 0 || a->rot_dims > a->dk || a->rot_dims % 2 || (a->rot_dims && !a->rot)) return kErrBadShape;
  if (!a->pos_ptr && (a->pos < 0 || a->pos + a->S > a->rot_rows)) return kErrBadShape;
  if (a->k_lin && a->hist + a->S > a->lin_rows) return kErrBadShape;
  if (!a->k_lin && a->S > a->ring) return kErrBadShape;
  if (a->k_pool && (a->pool <= 0 || a->pool >= a->ring)) return kErrBadShape;
  PrepParams p;
  p.p = a->p; p.ld = a->ld; p.oq = a->oq; p.ok = a->ok; p.ov = a->ov; p.gq = a->gq; p.gk = a->gk;
  p.rot = static_cast<const float2*>(a->rot); p.rot_v = static_cast<const float2*>(a->rot_v);
  p.q = a->q; p.k_ring = a->k_ring; p.v_ring = a->v_ring; p.k_lin = a->k_lin; p.v_lin = a->v_lin;
  p.k_pool = a->k_pool; p.v_pool = a->v_pool; p.pos_ptr = a->pos_ptr;
  p.B = a->B; p.S = a->S; p.H = a->H; p.G = a->G; p.dk = a->dk; p.dv = a->dv; p.whole = a->whole;
  p.rot_dims = a->rot_dims; p.ring = a->ring; p.lin_rows = a->lin_rows; p.hist = a->hist; p.pos = a->pos;
  p.rot_rows = a->rot_rows; p.pool = a->pool; p.pool_rows = a->pool_rows; p.eps = a->eps;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  bool vec = a->dk % 8 == 0 && a->dv % 8 == 0 && a->ld % 8 == 0 && a->oq % 8 == 0 && a->ok % 8 == 0 && a->ov % 8 == 0;
  for (const void* q : {a->p, (const void*)a->q, (const void*)a->k_ring, (const void*)a->v_ring, (const void*)a->k_lin,
                        (const void*)a->v_lin, a->gq, a->gk, (const void*)a->k_pool, (const void*)a->v_pool})
    vec = vec && al16(q);
  const size_t smem = ((size_t)(a->H + a->G) * (a->dk + 1)) * sizeof(float);
  if (smem > 200 * 1024) return kErrTooLarge;
  auto kern = a->f32 ? (vec ? qkv_prep_kernel<float, 8> : qkv_prep_kernel<float, 1>)
                     : (vec ? qkv_prep_kernel<__nv_bfloat16, 8> : qkv_prep_kernel<__nv_bfloat16, 1>);
  if (smem > 48 * 1024) DPTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  return counted(1, (int)launch_k(kern, dim3(a->B * a->S), dim3(kPrepThreads), smem, st, p));
}

struct DptbPoolArgs {
  const void* k; const void* v; void* k_pool; void* v_pool;
  long long k_batch, v_batch;
  int B, nk, nv, ring, lin0, pool, pool_rows, first, count, f32;
};

extern "C" int dptb_pool_blocks(const DptbPoolArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->count <= 0) return 0;
  if (a->pool <= 0 || a->first < 0 || a->first + a->count > a->pool_rows || a->B > 65535) return kErrBadShape;
  if (a->ring > 0 ? a->pool > a->ring : a->first * a->pool < a->lin0) return kErrBadShape;
  PoolParams p;
  p.k = a->k; p.v = a->v; p.k_batch = a->k_batch; p.v_batch = a->v_batch; p.k_pool = a->k_pool; p.v_pool = a->v_pool;
  p.nk = a->nk; p.nv = a->nv; p.ring = a->ring; p.lin0 = a->lin0; p.pool = a->pool; p.pool_rows = a->pool_rows;
  p.first = a->first;
  const dim3 grid(a->count, a->B);
  bool vec = a->nk % 8 == 0 && a->nv % 8 == 0 && a->k_batch % 8 == 0 && a->v_batch % 8 == 0;
  for (const void* q : {a->k, a->v, (const void*)a->k_pool, (const void*)a->v_pool})
    vec = vec && (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  auto kern = a->f32 ? (vec ? pool_blocks_kernel<float, 8> : pool_blocks_kernel<float, 1>)
                     : (vec ? pool_blocks_kernel<__nv_bfloat16, 8> : pool_blocks_kernel<__nv_bfloat16, 1>);
  return counted(1, (int)launch_k(kern, grid, dim3(kPoolThreads), (size_t)0, st, p));
}

struct DptbWindowArgs {
  const void* q; const void* k; const void* v; const void* k_pool; const void* v_pool; const void* sink; const void* rot_v;
  void* o; const int* pos_ptr;
  long long k_batch, v_batch;
  int B, S, H, G, dk, dv, ring, lin0, window, pool, pool_rows, pos, f32;
  float scale;
};

extern "C" int dptb_window_attn(const DptbWindowArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->S <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || a->H % a->G || a->dk <= 0 || a->dv <= 0 || a->window < 1 || a->H > 65535) return kErrBadShape;
  if (a->pool > 0 && (!a->k_pool || !a->v_pool)) return kErrBadShape;
  // a ring still holds every key of the first query's window after the last new row has been written
  if (a->ring > 0 && a->window + a->S - 1 > a->ring) return kErrBadShape;
  WindowParams p;
  p.q = a->q; p.k = a->k; p.v = a->v; p.k_pool = a->k_pool; p.v_pool = a->v_pool; p.sink = a->sink;
  p.rot_v = static_cast<const float2*>(a->rot_v); p.o = a->o; p.pos_ptr = a->pos_ptr;
  p.k_batch = a->k_batch; p.v_batch = a->v_batch;
  p.B = a->B; p.S = a->S; p.H = a->H; p.G = a->G; p.dk = a->dk; p.dv = a->dv; p.ring = a->ring; p.lin0 = a->lin0;
  p.window = a->window; p.pool = a->pool; p.pool_rows = a->pool_rows; p.pos = a->pos; p.scale = a->scale;
  return a->f32 ? launch_window<float>(p, st) : launch_window<__nv_bfloat16>(p, st);
}
