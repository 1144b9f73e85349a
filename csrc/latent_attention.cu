// Latent attention: keys and values are linear maps of one cached vector per token (the latent, R values), shared by all
// heads.  A head's score against token j is q . (Wk c_j) = (Wk^T q) . c_j, so with the query moved into latent space
// (q' = Wk^T q, one R-vector per head) the cache itself is both the keys and the values:
//   o'_h = sum_j softmax_j(scale * q'_h . c_j) c_j          and the head's output is Wv o'_h.
//
//   latent_norm_append   RMS norms of the two projections of a token (query latent, key/value latent); the latter goes
//                        straight into the cache row of its position
//   latent_attn_mma      bf16, R a multiple of 32 up to 512: one CTA serves 16 heads of one query and a slice of the keys.
//                        The cache rows stream through a two-stage cp.async ring; scores and weighted sums run on
//                        tensor-core fragments (heads are the 16 rows), which the 2 * 16 multiply-adds per cached byte
//                        pair need: CUDA cores could not keep up with HBM.  Scores, maxima, exponentials and sums are
//                        fp32, and the weights enter the second product as a high and a low bf16 part (16 mantissa bits).
//   latent_attn_merge    folds the key slices of a query
//   latent_attn_simt     any R and dtype (the fp32 path): one warp streams keys for one head
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

// ------------------------------------------------------------------------------------------- norms + cache append
struct LatentAppendParams {
  const void* d;            // [B*S, Rq + R] projections: query latent, then key/value latent
  long long ldd;
  const void* gq;           // [Rq]
  const void* gc;           // [R]
  void* cq;                 // [B*S, Rq]
  void* cache;              // [B, cap, R]
  void* c_new;              // optional dense copy [B*S, R]
  int B, S, Rq, R, cap, pos;
  const int* pos_ptr;       // device position (overrides pos)
  float eps;
};

// One warp per (token, projection); V consecutive features per lane and load, the first kKeep loads stay in registers.
template <typename T, int V>
__global__ void __launch_bounds__(128) latent_norm_append_kernel(const LatentAppendParams p) {
  constexpr int kKeep = V == 8 ? 3 : 4;
  const int wid = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int row = wid >> 1, which = wid & 1;
  const int n = which ? p.R : p.Rq;
  const T* g = static_cast<const T*>(which ? p.gc : p.gq);
  pdl_wait();
  pdl_launch_dependents();
  if (row >= p.B * p.S) return;
  const int pos0 = p.pos_ptr ? *p.pos_ptr : p.pos;
  const T* src = static_cast<const T*>(p.d) + (long long)row * p.ldd + (which ? p.Rq : 0);
  auto load = [&](const T* q, float (&o)[V]) {
    if constexpr (V == 8) Vec8<T>::load(q, o);
    else o[0] = to_f32(q[0]);
  };
  float v[kKeep][V], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (i * 32 + lane) * V;
#pragma unroll
    for (int k = 0; k < V; ++k) v[i][k] = 0.0f;
    if (c < n) load(src + c, v[i]);
  }
#pragma unroll
  for (int i = 0; i < kKeep; ++i)
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(v[i][k], v[i][k], ss);
  for (int c = (kKeep * 32 + lane) * V; c < n; c += 32 * V) {
    float t[V];
    load(src + c, t);
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(t[k], t[k], ss);
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)n + p.eps);
  T* dst;
  T* dst2 = nullptr;
  if (which) {
    const int b = row / p.S, at = pos0 + row % p.S;
    if (at < 0 || at >= p.cap) {
      if (lane == 0) report_error(kBadArgument);
      return;
    }
    dst = static_cast<T*>(p.cache) + ((long long)b * p.cap + at) * p.R;
    if (p.c_new) dst2 = static_cast<T*>(p.c_new) + (long long)row * p.R;
  } else {
    dst = static_cast<T*>(p.cq) + (long long)row * p.Rq;
  }
  auto put = [&](int c, const float (&x)[V]) {
    float w[V], o[V];
    load(g + c, w);
#pragma unroll
    for (int k = 0; k < V; ++k) o[k] = x[k] * inv * w[k];
    if constexpr (V == 8) {
      Vec8<T>::store(dst + c, o);
      if (dst2) Vec8<T>::store(dst2 + c, o);
    } else {
      dst[c] = from_f32<T>(o[0]);
      if (dst2) dst2[c] = from_f32<T>(o[0]);
    }
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (i * 32 + lane) * V;
    if (c < n) put(c, v[i]);
  }
  for (int c = (kKeep * 32 + lane) * V; c < n; c += 32 * V) {
    float t[V];
    load(src + c, t);
    put(c, t);
  }
}

// ------------------------------------------------------------------------------------------- attention
struct LatentAttnParams {
  const void* q;            // [B*S, H * R]
  const void* cache;        // [B, cap, R]
  void* o;                  // [B*S, H * R]
  int B, S, H, R, cap, pos;
  const int* pos_ptr;
  float scale;
  int splits;
  float* ws;                // [B*S][H][splits][R + 4]: sums, then maximum and weight sum
};

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

constexpr int kLaKeys = 32;       // keys per tile: four 8-key column tiles, each scored by two warps (half of R each)
constexpr int kLaThreads = 256;
constexpr int kLaPs = kLaKeys + 4;

__host__ __device__ inline int la_row_bytes(int R) { return R * 2 + 16; }   // padded: conflict-free ldmatrix rows
__host__ __device__ inline int la_smem_bytes(int R) {
  return (16 + 2 * kLaKeys) * la_row_bytes(R) + (2 * 16 * kLaPs + 16 * 3) * 4;
}

// MAXP: pairs of 8-column output tiles a warp holds (R / 16 pairs over 8 warps).
template <int MAXP>
__global__ void __launch_bounds__(kLaThreads)
latent_attn_mma_kernel(const LatentAttnParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int R = p.R, rb = la_row_bytes(R);
  uint8_t* qs = smem;
  uint8_t* cs = smem + 16 * rb;
  float* ps = reinterpret_cast<float*>(cs + 2 * kLaKeys * rb);   // [2][16][kLaPs]: score halves; plane 0 then the weights
  float* m_s = ps + 2 * 16 * kLaPs;                              // [16] running maximum
  float* l_s = m_s + 16;                                         // [16] running sum
  float* al_s = l_s + 16;                                        // [16] rescale of this tile

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, hg = blockIdx.y, row = blockIdx.z;
  const int b = row / p.S, sq = row % p.S;
  pdl_wait();
  pdl_launch_dependents();
  const int last = min((p.pos_ptr ? *p.pos_ptr : p.pos) + sq, p.cap - 1);   // last visible key
  const int n_tiles = last / kLaKeys + 1;
  const int per = (n_tiles + p.splits - 1) / p.splits;
  const int t0 = split * per, t1 = min(n_tiles, t0 + per);
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.cache) + (long long)b * p.cap * R;
  const int vpr = R / 8;                                         // 16-byte pieces of a row
  const int key_a = threadIdx.x / vpr, v_a = threadIdx.x % vpr;  // this thread's first piece of a tile ...
  const int key_d = kLaThreads / vpr, v_d = kLaThreads % vpr;    // ... and the step to the next

  auto load_tile = [&](int t, int stage) {
    const uint32_t dst = smem_u32(cs + stage * kLaKeys * rb);
    int key = key_a, v = v_a;
    while (key < kLaKeys) {
      const int j = t * kLaKeys + key;
      const bool ok = j <= last;
      cp_async_16(dst + key * rb + v * 16, cache + (long long)(ok ? j : last) * R + v * 8, ok);
      key += key_d;
      v += v_d;
      if (v >= vpr) {
        v -= vpr;
        ++key;
      }
    }
  };
  if (t0 < t1) load_tile(t0, 0);
  cp_async_commit();
  // the 16 heads' queries (rows past H are zero)
  for (int i = threadIdx.x; i < 16 * vpr; i += kLaThreads) {
    const int hh = i / vpr, v = i % vpr;
    const int h = hg * 16 + hh;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (h < p.H)
      u = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.q) + ((long long)row * p.H + h) * R + v * 8);
    *reinterpret_cast<uint4*>(qs + hh * rb + v * 16) = u;
  }
  if (threadIdx.x < 16) {
    m_s[threadIdx.x] = -INFINITY;
    l_s[threadIdx.x] = 0.0f;
  }
  float acc[MAXP][8];
#pragma unroll
  for (int n = 0; n < MAXP; ++n)
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[n][i] = 0.0f;
  const int pairs = R / 16;              // this warp's output columns: 16-column pairs warp, warp + 8, ...
  const float sl2 = p.scale * 1.4426950408889634f;
  const int nt = warp & 3, half = warp >> 2;      // scores: 8 keys, half of the features (R / 32 steps of 16)
  const uint32_t q_addr = smem_u32(qs) + (lane & 15) * rb + (lane >> 4) * 16 + half * R;
  const uint32_t k_off = (nt * 8 + (lane & 7)) * rb + (lane >> 3) * 16 + half * R;

  for (int t = t0; t < t1; ++t) {
    const int stage = (t - t0) & 1;
    if (t + 1 < t1) load_tile(t + 1, stage ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t ct = smem_u32(cs + stage * kLaKeys * rb);
    // ---- scores of 16 heads x 8 keys over half of R; four accumulators keep four products in flight
    float s[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) s[i][k] = 0.0f;
    const uint32_t kb = ct + k_off;
    int k = 0;
    for (; k + 4 <= R / 32; k += 4) {
      uint32_t a[4][4], bb[2][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) ldmatrix_x4(a[i], q_addr + (k + i) * 32);
      ldmatrix_x4(bb[0], kb + k * 32);
      ldmatrix_x4(bb[1], kb + (k + 2) * 32);
#pragma unroll
      for (int i = 0; i < 4; ++i) mma_bf16_16816(s[i], a[i], bb[i >> 1][(i & 1) * 2], bb[i >> 1][(i & 1) * 2 + 1]);
    }
    for (; k < R / 32; ++k) {            // (the upper half of the loaded key fragment belongs to the next step)
      uint32_t a[4], bb[4];
      ldmatrix_x4(a, q_addr + k * 32);
      ldmatrix_x4(bb, kb + k * 32);
      mma_bf16_16816(s[0], a, bb[0], bb[1]);
    }
    {
      const int r0 = lane >> 2, c0 = nt * 8 + (lane & 3) * 2;
      float* pr = ps + half * 16 * kLaPs + r0 * kLaPs + c0;
      *reinterpret_cast<float2*>(pr) =
          make_float2((s[0][0] + s[1][0]) + (s[2][0] + s[3][0]), (s[0][1] + s[1][1]) + (s[2][1] + s[3][1]));
      *reinterpret_cast<float2*>(pr + 8 * kLaPs) =
          make_float2((s[0][2] + s[1][2]) + (s[2][2] + s[3][2]), (s[0][3] + s[1][3]) + (s[2][3] + s[3][3]));
    }
    __syncthreads();
    // ---- softmax: 16 threads per head, 2 keys each (a head's threads are neighbours in one warp)
    {
      const int hh = threadIdx.x >> 4, c0 = (threadIdx.x & 15) * 2;
      float* pr = ps + hh * kLaPs + c0;
      const float2 x = *reinterpret_cast<const float2*>(pr);
      const float2 y = *reinterpret_cast<const float2*>(pr + 16 * kLaPs);
      const int j = t * kLaKeys + c0;
      const float v0 = j <= last ? (x.x + y.x) * sl2 : -INFINITY;
      const float v1 = j + 1 <= last ? (x.y + y.y) * sl2 : -INFINITY;
      float mx = fmaxf(v0, v1);
#pragma unroll
      for (int o = 1; o < 16; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = m_s[hh];
      const float m_new = fmaxf(m_old, mx);       // finite: every tile in range has a visible key
      const float w0 = exp2f(v0 - m_new), w1 = exp2f(v1 - m_new);
      *reinterpret_cast<float2*>(pr) = make_float2(w0, w1);
      float sum = w0 + w1;
#pragma unroll
      for (int o = 1; o < 16; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if ((threadIdx.x & 15) == 0) {              // (the shuffles above order every lane's read of m_s before this)
        const float al = exp2f(m_old - m_new);
        al_s[hh] = al;
        m_s[hh] = m_new;
        l_s[hh] = l_s[hh] * al + sum;
      }
    }
    __syncthreads();
    // ---- o' += P C over this warp's columns, weights as high + low bf16 parts
    {
      const int r0 = lane >> 2;
      const float al0 = al_s[r0], al1 = al_s[r0 + 8];
      if (__any_sync(0xffffffffu, al0 != 1.0f || al1 != 1.0f)) {
#pragma unroll
        for (int n = 0; n < MAXP; ++n) {
          acc[n][0] *= al0; acc[n][1] *= al0; acc[n][4] *= al0; acc[n][5] *= al0;
          acc[n][2] *= al1; acc[n][3] *= al1; acc[n][6] *= al1; acc[n][7] *= al1;
        }
      }
#pragma unroll
      for (int kk = 0; kk < kLaKeys / 16; ++kk) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {     // fragment register i: row + 8 * (i & 1), keys + 8 * (i >> 1)
          const float2 w = *reinterpret_cast<const float2*>(ps + (r0 + 8 * (i & 1)) * kLaPs + kk * 16 + 8 * (i >> 1) +
                                                            (lane & 3) * 2);
          hi[i] = pack_bf16x2(w.x, w.y);
          const float2 h = unpack_bf16x2(hi[i]);
          lo[i] = pack_bf16x2(w.x - h.x, w.y - h.y);
        }
        // lanes 0-15: the 16 keys' first 8 columns, lanes 16-31: the next 8
        const uint32_t vb = ct + (kk * 16 + (lane & 15)) * rb + (lane >> 4) * 16;
#pragma unroll
        for (int n = 0; n < MAXP; ++n) {
          const int pr = warp + n * 8;
          if (pr < pairs) {
            uint32_t bv[4];
            ldmatrix_x4_trans(bv, vb + pr * 32);
            float(&d0)[4] = *reinterpret_cast<float(*)[4]>(&acc[n][0]);
            float(&d1)[4] = *reinterpret_cast<float(*)[4]>(&acc[n][4]);
            mma_bf16_16816(d0, hi, bv[0], bv[1]);
            mma_bf16_16816(d1, hi, bv[2], bv[3]);
            mma_bf16_16816(d0, lo, bv[0], bv[1]);
            mma_bf16_16816(d1, lo, bv[2], bv[3]);
          }
        }
      }
    }
    __syncthreads();      // the tile and the weights may be overwritten
  }
  cp_async_wait<0>();
  __syncthreads();

  const int r0 = lane >> 2;
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    const int hh = r0 + hr * 8, h = hg * 16 + hh;
    if (h >= p.H) continue;
    if (p.splits == 1) {
      const float inv = 1.0f / l_s[hh];
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.o) + ((long long)row * p.H + h) * R;
#pragma unroll
      for (int n = 0; n < MAXP; ++n) {
        const int pr = warp + n * 8;
        if (pr >= pairs) continue;
        const int c = pr * 16 + (lane & 3) * 2;
        *reinterpret_cast<uint32_t*>(out + c) = pack_bf16x2(acc[n][hr * 2] * inv, acc[n][hr * 2 + 1] * inv);
        *reinterpret_cast<uint32_t*>(out + c + 8) = pack_bf16x2(acc[n][4 + hr * 2] * inv, acc[n][4 + hr * 2 + 1] * inv);
      }
    } else {
      float* mine = p.ws + (((long long)row * p.H + h) * p.splits + split) * (R + 4);
#pragma unroll
      for (int n = 0; n < MAXP; ++n) {
        const int pr = warp + n * 8;
        if (pr >= pairs) continue;
        const int c = pr * 16 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(mine + c) = make_float2(acc[n][hr * 2], acc[n][hr * 2 + 1]);
        *reinterpret_cast<float2*>(mine + c + 8) = make_float2(acc[n][4 + hr * 2], acc[n][4 + hr * 2 + 1]);
      }
      if (warp == 0 && (lane & 3) == 0) {
        mine[R] = m_s[hh];
        mine[R + 1] = l_s[hh];
      }
    }
  }
}

// One CTA per (query, head): o' = sum over slices of 2^(m_s - m) x_s / sum of the rescaled weight sums.
__global__ void __launch_bounds__(128) latent_attn_merge_kernel(const LatentAttnParams p) {
  __shared__ float wt[64];
  __shared__ float inv_s;
  const int R = p.R, st = R + 4;
  pdl_wait();
  pdl_launch_dependents();
  const long long rh = blockIdx.x;
  const float* base = p.ws + rh * p.splits * st;
  if (threadIdx.x < 32) {
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
    if (s0 < p.splits) { m0 = __ldcg(base + s0 * st + R); l0 = __ldcg(base + s0 * st + R + 1); }
    if (s1 < p.splits) { m1 = __ldcg(base + s1 * st + R); l1 = __ldcg(base + s1 * st + R + 1); }
    const float m = warp_max(fmaxf(m0, m1));
    const float w0 = exp2f(m0 - m), w1 = exp2f(m1 - m);      // an empty slice has maximum -inf: weight 0
    const float l = warp_sum(l0 * w0 + l1 * w1);
    wt[s0] = w0;
    wt[s1] = w1;
    if (threadIdx.x == 0) inv_s = 1.0f / l;
  }
  __syncthreads();
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.o) + rh * R;
  for (int c = threadIdx.x * 4; c < R; c += 512) {
    float x[4] = {0, 0, 0, 0};
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float4 v = __ldcg(reinterpret_cast<const float4*>(base + s * st + c));
      const float w = wt[s];
      x[0] = fmaf(v.x, w, x[0]); x[1] = fmaf(v.y, w, x[1]);
      x[2] = fmaf(v.z, w, x[2]); x[3] = fmaf(v.w, w, x[3]);
    }
    const float inv = inv_s;
    *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16x2(x[0] * inv, x[1] * inv), pack_bf16x2(x[2] * inv, x[3] * inv));
  }
}

// Generic form: a CTA of 4 warps per (query, head); every warp takes every fourth key with its own running softmax, the
// four are folded at the end.  MAXV * 32 >= R.
template <typename T, int MAXV>
__global__ void __launch_bounds__(128) latent_attn_simt_kernel(const LatentAttnParams p) {
  __shared__ float red[4][MAXV * 32 + 2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, row = blockIdx.y;
  const int b = row / p.S, sq = row % p.S, R = p.R;
  pdl_wait();
  pdl_launch_dependents();
  const int last = min((p.pos_ptr ? *p.pos_ptr : p.pos) + sq, p.cap - 1);
  const T* q = static_cast<const T*>(p.q) + ((long long)row * p.H + h) * R;
  const T* cache = static_cast<const T*>(p.cache) + (long long)b * p.cap * R;
  float qv[MAXV], o[MAXV];
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = i * 32 + lane;
    qv[i] = c < R ? to_f32(q[c]) : 0.0f;
    o[i] = 0.0f;
  }
  float m = -INFINITY, l = 0.0f;
  for (int j = warp; j <= last; j += 4) {
    const T* k = cache + (long long)j * R;
    float kv[MAXV], s = 0.0f;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = i * 32 + lane;
      kv[i] = c < R ? to_f32(k[c]) : 0.0f;
      s = fmaf(qv[i], kv[i], s);
    }
    s = warp_sum(s) * p.scale;
    const float m_new = fmaxf(m, s);
    const float al = expf(m - m_new), w = expf(s - m_new);
    l = l * al + w;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) o[i] = fmaf(w, kv[i], o[i] * al);
    m = m_new;
  }
#pragma unroll
  for (int i = 0; i < MAXV; ++i) red[warp][i * 32 + lane] = o[i];
  if (lane == 0) {
    red[warp][MAXV * 32] = m;
    red[warp][MAXV * 32 + 1] = l;
  }
  __syncthreads();
  float mm = -INFINITY, ll = 0.0f, wt[4];
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, red[w][MAXV * 32]);
  for (int w = 0; w < 4; ++w) {
    wt[w] = expf(red[w][MAXV * 32] - mm);
    ll += red[w][MAXV * 32 + 1] * wt[w];
  }
  const float inv = 1.0f / ll;
  T* out = static_cast<T*>(p.o) + ((long long)row * p.H + h) * R;
  for (int c = threadIdx.x; c < R; c += 128) {
    float v = 0.0f;
    for (int w = 0; w < 4; ++w) v += red[w][c] * wt[w];
    out[c] = from_f32<T>(v * inv);
  }
}

template <int MAXP>
static int launch_latent_mma(const LatentAttnParams& p, dim3 grid, cudaStream_t st) {
  auto kern = latent_attn_mma_kernel<MAXP>;
  const int bytes = la_smem_bytes(p.R);
  static int configured = 0;
  if (configured < bytes) {
    DPTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    configured = bytes;
  }
  const int rc = counted(1, (int)launch_k(kern, grid, dim3(kLaThreads), (size_t)bytes, st, p));
  if (rc || p.splits == 1) return rc;
  return counted(1, (int)launch_k(latent_attn_merge_kernel, dim3((unsigned)(p.B * p.S * p.H)), dim3(128), (size_t)0, st, p));
}
template <typename T>
static int launch_latent_simt(const LatentAttnParams& p, cudaStream_t st) {
  const dim3 grid(p.H, p.B * p.S);
  if (p.R <= 64) return counted(1, (int)launch_k(latent_attn_simt_kernel<T, 2>, grid, dim3(128), (size_t)0, st, p));
  if (p.R <= 128) return counted(1, (int)launch_k(latent_attn_simt_kernel<T, 4>, grid, dim3(128), (size_t)0, st, p));
  if (p.R <= 256) return counted(1, (int)launch_k(latent_attn_simt_kernel<T, 8>, grid, dim3(128), (size_t)0, st, p));
  if (p.R <= 512) return counted(1, (int)launch_k(latent_attn_simt_kernel<T, 16>, grid, dim3(128), (size_t)0, st, p));
  if (p.R <= 1024) return counted(1, (int)launch_k(latent_attn_simt_kernel<T, 32>, grid, dim3(128), (size_t)0, st, p));
  return kErrUnsupported;
}

}  // namespace dptb

using namespace dptb;

struct DptbLatentArgs {
  const void* d; const void* gq; const void* gc; void* cq; void* c_new;      // append
  const void* q; void* o; float* ws;                                         // attention
  void* cache;
  const int* pos_ptr;
  long long ldd, ws_floats;
  int B, S, H, Rq, R, cap, pos, splits, f32, force_simt;
  float eps, scale;
};

extern "C" int dptb_latent_norm_append(const DptbLatentArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->S <= 0) return 0;
  if (a->Rq <= 0 || a->R <= 0 || a->ldd < a->Rq + a->R) return kErrBadShape;
  if (!a->pos_ptr && (a->pos < 0 || a->pos + a->S > a->cap)) return kErrBadShape;
  LatentAppendParams p;
  p.d = a->d; p.ldd = a->ldd; p.gq = a->gq; p.gc = a->gc; p.cq = a->cq; p.cache = a->cache; p.c_new = a->c_new;
  p.B = a->B; p.S = a->S; p.Rq = a->Rq; p.R = a->R; p.cap = a->cap; p.pos = a->pos; p.pos_ptr = a->pos_ptr; p.eps = a->eps;
  const dim3 grid((2 * a->B * a->S + 3) / 4);
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = a->Rq % 8 == 0 && a->R % 8 == 0 && a->ldd % 8 == 0 && al16(a->d) && al16(a->gq) && al16(a->gc) &&
                   al16(a->cq) && al16(a->cache) && (!a->c_new || al16(a->c_new));
  auto kern = a->f32 ? (vec ? latent_norm_append_kernel<float, 8> : latent_norm_append_kernel<float, 1>)
                     : (vec ? latent_norm_append_kernel<__nv_bfloat16, 8> : latent_norm_append_kernel<__nv_bfloat16, 1>);
  return counted(1, (int)launch_k(kern, grid, dim3(128), (size_t)0, st, p));
}

static bool latent_mma_ok(int R, int f32) { return !f32 && R % 32 == 0 && R <= 512; }

// Key slices per query: enough CTAs to fill the SMs, at least four key tiles each at the largest context.
extern "C" int dptb_latent_attn_splits(int rows, int H, int R, int max_keys, int f32) {
  if (!latent_mma_ok(R, f32)) return 1;
  const int groups = rows * ((H + 15) / 16);
  int s = (sm_count() * 2) / (groups > 0 ? groups : 1);
  const int by_keys = (max_keys + 4 * kLaKeys - 1) / (4 * kLaKeys);
  if (s > by_keys) s = by_keys;
  if (s > 64) s = 64;
  return s < 1 ? 1 : s;
}
extern "C" long long dptb_latent_attn_ws_floats(int rows, int H, int R, int splits) {
  return splits <= 1 ? 0 : (long long)rows * H * splits * (R + 4);
}

extern "C" int dptb_latent_attn(const DptbLatentArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  const int rows = a->B * a->S;
  if (rows <= 0) return 0;
  if (a->H <= 0 || a->R <= 0) return kErrBadShape;
  if (!a->pos_ptr && (a->pos < 0 || a->pos + a->S > a->cap)) return kErrBadShape;
  LatentAttnParams p;
  p.q = a->q; p.cache = a->cache; p.o = a->o;
  p.B = a->B; p.S = a->S; p.H = a->H; p.R = a->R; p.cap = a->cap; p.pos = a->pos; p.pos_ptr = a->pos_ptr;
  p.scale = a->scale; p.splits = a->splits < 1 ? 1 : a->splits; p.ws = a->ws;
  if (rows > 65535) return kErrTooLarge;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (!a->force_simt && latent_mma_ok(a->R, a->f32) && al16(a->q) && al16(a->cache) && al16(a->o)) {
    const int hg = (a->H + 15) / 16;
    if (p.splits > 64 || (p.splits > 1 && (!a->ws || !al16(a->ws) ||
                                           dptb_latent_attn_ws_floats(rows, a->H, a->R, p.splits) > a->ws_floats)))
      return kErrTooLarge;
    const dim3 grid(p.splits, hg, rows);
    if (a->R <= 128) return launch_latent_mma<1>(p, grid, st);
    if (a->R <= 256) return launch_latent_mma<2>(p, grid, st);
    return launch_latent_mma<4>(p, grid, st);
  }
  return a->f32 ? launch_latent_simt<float>(p, st) : launch_latent_simt<__nv_bfloat16>(p, st);
}
