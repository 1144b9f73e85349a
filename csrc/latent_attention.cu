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
//                        The last CTA of a query folds the key slices.
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

// One warp per (token, projection).
template <typename T>
__global__ void __launch_bounds__(128) latent_norm_append_kernel(const LatentAppendParams p) {
  const int wid = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  const int row = wid >> 1, which = wid & 1;
  if (row >= p.B * p.S) return;
  const int n = which ? p.R : p.Rq;
  const T* src = static_cast<const T*>(p.d) + (long long)row * p.ldd + (which ? p.Rq : 0);
  const T* g = static_cast<const T*>(which ? p.gc : p.gq);
  float ss = 0.0f;
  for (int i = lane; i < n; i += 32) {
    const float v = to_f32(src[i]);
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)n + p.eps);
  T* dst;
  T* dst2 = nullptr;
  if (which) {
    const int b = row / p.S, s = row % p.S;
    const int at = (p.pos_ptr ? *p.pos_ptr : p.pos) + s;
    if (at < 0 || at >= p.cap) {
      if (lane == 0) report_error(kBadArgument);
      return;
    }
    dst = static_cast<T*>(p.cache) + ((long long)b * p.cap + at) * p.R;
    if (p.c_new) dst2 = static_cast<T*>(p.c_new) + (long long)row * p.R;
  } else {
    dst = static_cast<T*>(p.cq) + (long long)row * p.Rq;
  }
  for (int i = lane; i < n; i += 32) {
    const T v = from_f32<T>(to_f32(src[i]) * inv * to_f32(g[i]));
    dst[i] = v;
    if (dst2) dst2[i] = v;
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
  float* ws;                // [B*S * ceil(H/16)][splits][16][R + 2]
  int* counters;            // [B*S * ceil(H/16)], zero between launches
};

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t (&r)[2], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t (&r)[2], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

constexpr int kLaKeys = 64;       // keys per tile; each of the 4 warps scores 16 of them
constexpr int kLaThreads = 128;

__host__ __device__ inline int la_row_bytes(int R) { return R * 2 + 16; }   // padded: conflict-free ldmatrix rows
__host__ __device__ inline int la_smem_bytes(int R) {
  return (16 + 2 * kLaKeys) * la_row_bytes(R) + (16 * (kLaKeys + 4) + 16 * 3 + 4) * 4;
}

// MAXNT: 8-column tiles of the R output columns a warp can hold (R / 32 <= MAXNT).
template <int MAXNT>
__global__ void __launch_bounds__(kLaThreads)
latent_attn_mma_kernel(const LatentAttnParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int R = p.R, rb = la_row_bytes(R);
  uint8_t* qs = smem;
  uint8_t* cs = smem + 16 * rb;
  float* ps = reinterpret_cast<float*>(cs + 2 * kLaKeys * rb);   // [16][kLaKeys + 4] scores, then weights
  float* m_s = ps + 16 * (kLaKeys + 4);                          // [16] running maximum
  float* l_s = m_s + 16;                                         // [16] running sum
  float* al_s = l_s + 16;                                        // [16] rescale of this tile
  int* flag_s = reinterpret_cast<int*>(al_s + 16);

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
  const int vec_per_row = R / 8;

  auto load_tile = [&](int t, int stage) {
    uint8_t* dst = cs + stage * kLaKeys * rb;
    for (int i = threadIdx.x; i < kLaKeys * vec_per_row; i += kLaThreads) {
      const int key = i / vec_per_row, v = i % vec_per_row;
      const int j = t * kLaKeys + key;
      const bool ok = j <= last;
      cp_async_16(smem_u32(dst + key * rb + v * 16), cache + (long long)(ok ? j : last) * R + v * 8, ok);
    }
  };
  if (t0 < t1) load_tile(t0, 0);
  cp_async_commit();
  // the 16 heads' queries (rows past H are zero)
  for (int i = threadIdx.x; i < 16 * vec_per_row; i += kLaThreads) {
    const int hh = i / vec_per_row, v = i % vec_per_row;
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
  float acc[MAXNT][4];
#pragma unroll
  for (int n = 0; n < MAXNT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[n][i] = 0.0f;
  const int nt = R / 32;                 // this warp's output columns: [warp * 8 * nt, + 8 * nt)
  const float sl2 = p.scale * 1.4426950408889634f;

  for (int t = t0; t < t1; ++t) {
    const int stage = (t - t0) & 1;
    if (t + 1 < t1) load_tile(t + 1, stage ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint8_t* ct = cs + stage * kLaKeys * rb;
    // ---- scores of 16 heads x 16 keys
    float s0[4] = {0, 0, 0, 0}, s1[4] = {0, 0, 0, 0};
    const uint32_t qa = smem_u32(qs + (lane & 15) * rb + (lane >> 4) * 16);
    const uint32_t kb = smem_u32(ct + (warp * 16 + (lane & 7)) * rb + ((lane >> 3) & 1) * 16);
    for (int k = 0; k < R / 16; ++k) {
      uint32_t a[4], b0[2], b1[2];
      ldmatrix_x4(a, qa + k * 32);
      ldmatrix_x2(b0, kb + k * 32);
      ldmatrix_x2(b1, kb + 8 * rb + k * 32);
      mma_bf16_16816(s0, a, b0);
      mma_bf16_16816(s1, a, b1);
    }
    {
      const int r0 = lane >> 2, c0 = warp * 16 + (lane & 3) * 2;
      const int j0 = t * kLaKeys + c0;
      float* pr0 = ps + r0 * (kLaKeys + 4);
      float* pr1 = ps + (r0 + 8) * (kLaKeys + 4);
      pr0[c0] = j0 <= last ? s0[0] * sl2 : -INFINITY;
      pr0[c0 + 1] = j0 + 1 <= last ? s0[1] * sl2 : -INFINITY;
      pr1[c0] = j0 <= last ? s0[2] * sl2 : -INFINITY;
      pr1[c0 + 1] = j0 + 1 <= last ? s0[3] * sl2 : -INFINITY;
      pr0[c0 + 8] = j0 + 8 <= last ? s1[0] * sl2 : -INFINITY;
      pr0[c0 + 9] = j0 + 9 <= last ? s1[1] * sl2 : -INFINITY;
      pr1[c0 + 8] = j0 + 8 <= last ? s1[2] * sl2 : -INFINITY;
      pr1[c0 + 9] = j0 + 9 <= last ? s1[3] * sl2 : -INFINITY;
    }
    __syncthreads();
    // ---- softmax: 8 threads per head, 8 keys each (a head's 8 threads are neighbours in one warp)
    {
      const int hh = threadIdx.x >> 3, part = threadIdx.x & 7;
      float* pr = ps + hh * (kLaKeys + 4) + part * 8;
      float v[8], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        v[i] = pr[i];
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = m_s[hh];
      const float m_new = fmaxf(m_old, mx);       // finite: every tile in range has a visible key
      float sum = 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        v[i] = exp2f(v[i] - m_new);
        pr[i] = v[i];
        sum += v[i];
      }
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      __syncwarp();
      if (part == 0) {
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
#pragma unroll
      for (int n = 0; n < MAXNT; ++n) {
        acc[n][0] *= al0; acc[n][1] *= al0;
        acc[n][2] *= al1; acc[n][3] *= al1;
      }
#pragma unroll
      for (int k = 0; k < kLaKeys / 16; ++k) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {     // fragment register i: row + 8 * (i & 1), keys + 8 * (i >> 1)
          const float2 w = *reinterpret_cast<const float2*>(ps + (r0 + 8 * (i & 1)) * (kLaKeys + 4) + k * 16 +
                                                            8 * (i >> 1) + (lane & 3) * 2);
          hi[i] = pack_bf16x2(w.x, w.y);
          const float2 h = unpack_bf16x2(hi[i]);
          lo[i] = pack_bf16x2(w.x - h.x, w.y - h.y);
        }
        const uint32_t vb = smem_u32(ct + (k * 16 + (lane & 15)) * rb + warp * 16 * nt);
#pragma unroll
        for (int n = 0; n < MAXNT; ++n) {
          if (n < nt) {
            uint32_t bv[2];
            ldmatrix_x2_trans(bv, vb + n * 16);
            mma_bf16_16816(acc[n], hi, bv);
            mma_bf16_16816(acc[n], lo, bv);
          }
        }
      }
    }
    __syncthreads();      // the tile and the weights may be overwritten
  }
  cp_async_wait<0>();

  const int r0 = lane >> 2;
  const int group = row * gridDim.y + hg;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.o) + (long long)row * p.H * R;
  if (p.splits == 1) {
    const float i0 = 1.0f / l_s[r0], i1 = 1.0f / l_s[r0 + 8];
    const int h0 = hg * 16 + r0, h1 = h0 + 8;
#pragma unroll
    for (int n = 0; n < MAXNT; ++n) {
      if (n < nt) {
        const int c = (warp * nt + n) * 8 + (lane & 3) * 2;
        if (h0 < p.H) *reinterpret_cast<uint32_t*>(out + (long long)h0 * R + c) = pack_bf16x2(acc[n][0] * i0, acc[n][1] * i0);
        if (h1 < p.H) *reinterpret_cast<uint32_t*>(out + (long long)h1 * R + c) = pack_bf16x2(acc[n][2] * i1, acc[n][3] * i1);
      }
    }
    return;
  }
  // ---- partials, and the fold by the CTA that arrives last
  const int st = R + 2;
  float* mine = p.ws + ((long long)group * p.splits + split) * 16 * st;
#pragma unroll
  for (int n = 0; n < MAXNT; ++n) {
    if (n < nt) {
      const int c = (warp * nt + n) * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(mine + r0 * st + c) = make_float2(acc[n][0], acc[n][1]);
      *reinterpret_cast<float2*>(mine + (r0 + 8) * st + c) = make_float2(acc[n][2], acc[n][3]);
    }
  }
  __syncthreads();
  if (threadIdx.x < 16) {
    mine[threadIdx.x * st + R] = m_s[threadIdx.x];
    mine[threadIdx.x * st + R + 1] = l_s[threadIdx.x];
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    const int old = atomicAdd(&p.counters[group], 1);
    *flag_s = old == p.splits - 1;
    if (old == p.splits - 1) p.counters[group] = 0;
  }
  __syncthreads();
  if (!*flag_s) return;
  __threadfence();
  const float* base = p.ws + (long long)group * p.splits * 16 * st;
  for (int i = threadIdx.x; i < 16 * (R / 2); i += kLaThreads) {
    const int hh = i / (R / 2), c = (i % (R / 2)) * 2;
    const int h = hg * 16 + hh;
    if (h >= p.H) continue;
    float m = -INFINITY;
    for (int s = 0; s < p.splits; ++s) m = fmaxf(m, __ldcg(base + (s * 16 + hh) * st + R));
    float l = 0.0f, x = 0.0f, y = 0.0f;
    for (int s = 0; s < p.splits; ++s) {
      const float* q = base + (s * 16 + hh) * st;
      const float w = exp2f(__ldcg(q + R) - m);       // an empty slice has maximum -inf: weight 0
      const float2 v = __ldcg(reinterpret_cast<const float2*>(q + c));
      l = fmaf(__ldcg(q + R + 1), w, l);
      x = fmaf(v.x, w, x);
      y = fmaf(v.y, w, y);
    }
    const float inv = 1.0f / l;
    *reinterpret_cast<uint32_t*>(out + (long long)h * R + c) = pack_bf16x2(x * inv, y * inv);
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

template <int MAXNT>
static int launch_latent_mma(const LatentAttnParams& p, dim3 grid, cudaStream_t st) {
  auto kern = latent_attn_mma_kernel<MAXNT>;
  const int bytes = la_smem_bytes(p.R);
  static int configured = 0;
  if (configured < bytes) {
    DPTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    configured = bytes;
  }
  return counted(1, (int)launch_k(kern, grid, dim3(kLaThreads), (size_t)bytes, st, p));
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
  const void* q; void* o; float* ws; int* counters;                          // attention
  void* cache;
  const int* pos_ptr;
  long long ldd, ws_floats;
  int B, S, H, Rq, R, cap, pos, splits, num_counters, f32, force_simt;
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
  return counted(1, (int)(a->f32 ? launch_k(latent_norm_append_kernel<float>, grid, dim3(128), (size_t)0, st, p)
                                 : launch_k(latent_norm_append_kernel<__nv_bfloat16>, grid, dim3(128), (size_t)0, st, p)));
}

static bool latent_mma_ok(int R, int f32) { return !f32 && R % 32 == 0 && R <= 512; }

// Key slices per query: enough CTAs to fill the SMs, at least two key tiles each at the largest context.
extern "C" int dptb_latent_attn_splits(int rows, int H, int R, int max_keys, int f32) {
  if (!latent_mma_ok(R, f32)) return 1;
  const int groups = rows * ((H + 15) / 16);
  const int per_sm = la_smem_bytes(R) <= 100 * 1024 ? 2 : 1;
  int s = (sm_count() * per_sm) / (groups > 0 ? groups : 1);
  const int by_keys = (max_keys + 2 * kLaKeys - 1) / (2 * kLaKeys);
  if (s > by_keys) s = by_keys;
  if (s > 64) s = 64;
  return s < 1 ? 1 : s;
}
extern "C" long long dptb_latent_attn_ws_floats(int rows, int H, int R, int splits) {
  return splits <= 1 ? 0 : (long long)rows * ((H + 15) / 16) * splits * 16 * (R + 2);
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
  p.scale = a->scale; p.splits = a->splits < 1 ? 1 : a->splits; p.ws = a->ws; p.counters = a->counters;
  if (rows > 65535) return kErrTooLarge;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (!a->force_simt && latent_mma_ok(a->R, a->f32) && al16(a->q) && al16(a->cache) && al16(a->o)) {
    const int hg = (a->H + 15) / 16;
    if (p.splits > 1 && (!a->ws || !a->counters || rows * hg > a->num_counters ||
                         dptb_latent_attn_ws_floats(rows, a->H, a->R, p.splits) > a->ws_floats))
      return kErrTooLarge;
    const dim3 grid(p.splits, hg, rows);
    const int nt = a->R / 32;
    if (nt <= 2) return launch_latent_mma<2>(p, grid, st);
    if (nt <= 4) return launch_latent_mma<4>(p, grid, st);
    if (nt <= 8) return launch_latent_mma<8>(p, grid, st);
    return launch_latent_mma<16>(p, grid, st);
  }
  return a->f32 ? launch_latent_simt<float>(p, st) : launch_latent_simt<__nv_bfloat16>(p, st);
}
