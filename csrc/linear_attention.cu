// Linear attention with a matrix state per head and a decay in front of it:
//
//   S_t = diag(a_t) S_{t-1} + k_t v_t^T          S [dk, dv] fp32, zero before the first token
//   o_t = S_t^T q_t
//
// a_t is either one number per key channel and token, a = sigmoid(z)^(1 / tau) with z = W2 r + b from a low-rank projection r
// of the token (gated linear attention), or one constant per head (lightning attention).  q, k and v are column ranges of one
// projected row; an activation and the query's scale are applied where they are read.
//
//   linear_step      token by token, exact recurrence, any dtype and size: decode steps, short inputs, fp32.  The decay enters
//                    as a - 1 = expm1(log a), so that long memories do not drift.
//   decay_kernel     running sums of log2 a over blocks of 64 tokens of a long input
//   linear_chunk     bf16, long inputs: pieces of up to 64 tokens as matrix products.  With G the running sum of log a inside
//                    a piece and G_1 its value at the piece's first token,
//                        o_i  = (q_i e^{G_i - G_1})^T (e^{G_1} S) + sum_{j <= i} (q_i e^{G_i - G_1}) . (k_j e^{G_1 - G_j}) v_j
//                        S'   = e^{G_end - G_1} (e^{G_1} S + sum_j (k_j e^{G_1 - G_j}) v_j^T)
//                    Every operand that carries a decay or the state enters the tensor core as a high and a low bf16 part (16
//                    mantissa bits), the state itself stays in fp32 registers.  A piece whose decays span more than 2^72 is
//                    cut shorter (down to one token, where the span is zero), so no factor overflows.
//                    The sequence is cut into segments that run in parallel: pass 1 finds what each segment adds to the state,
//                    pass 2 folds the segments before its own and computes outputs.
//   head_norm_gate   rms(o) * w * act(g): the norm over every head (one w for all) or over all heads together
#include <cuda_bf16.h>

#include "common/host.h"
#include "common/ptx.cuh"
#include "common/reduce.cuh"

namespace dptb {

struct LinearParams {
  const void* p;            // [B*S, ld] projected rows
  long long ld;
  int oq, ok, ov, orank;    // column of the queries, keys, values and low-rank decay inputs
  const void* w2;           // [H * dk, rank] (null: constant decay)
  const void* b2;           // [H * dk]
  const float* decay;       // [H, 2]: log a, a - 1
  float* log_a;             // [B*S, H * dk] (long inputs): log2 a summed from the start of the token's block of 64
  float* state;             // [B, H, dk, dv]
  void* o;                  // [B*S, H * dv]
  float* ends;              // [B, H, segments + 1, dk, dv]: state a segment adds; the last entry copies the initial state
  float* totals;            // [B, H, segments, dk]: decay over a segment, minus one
  int B, S, H, dk, dv, rank, silu, segments, seg_tokens;
  float q_scale, inv_tau;
};

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float fast_silu_f(float v) { return __fdividef(v, 1.0f + __expf(-v)); }    // bf16 results
// log sigmoid(z)
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

template <typename T>
__device__ __forceinline__ float low_rank_log_decay(const LinearParams& p, long long row, int hc) {
  const T* r = static_cast<const T*>(p.p) + row * p.ld + p.orank;
  const T* w = static_cast<const T*>(p.w2) + (long long)hc * p.rank;
  float z = to_f32(static_cast<const T*>(p.b2)[hc]);
  for (int i = 0; i < p.rank; ++i) z = fmaf(to_f32(w[i]), to_f32(r[i]), z);
  return log_sigmoid_f(z) * p.inv_tau;
}

// ------------------------------------------------------------------------------------------- token by token
constexpr int kStepThreads = 256;
constexpr int kStepCols = 16;       // column groups of V values
constexpr int kStepRows = 16;       // row groups; a thread holds rows rg, rg + 16, ...

template <typename T, int V, int NR>
__global__ void __launch_bounds__(kStepThreads) linear_step_kernel(const LinearParams p) {
  extern __shared__ float step_smem[];
  const int dk = p.dk, dv = p.dv;
  float* qs = step_smem;
  float* ks = qs + dk;
  float* es = ks + dk;              // a - 1
  float* red = es + dk;             // [8][kStepCols * V]
  const int cg = threadIdx.x & (kStepCols - 1), rg = threadIdx.x / kStepCols;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z;
  const int c0 = (blockIdx.x * kStepCols + cg) * V;
  const bool live = c0 < dv;
  // the state was written by an earlier step, several launches ago: it can be fetched before the wait
  float* state = p.state + ((long long)b * p.H + h) * dk * dv + c0;
  float S[NR][V];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = rg + kStepRows * i;
#pragma unroll
    for (int k = 0; k < V; ++k) S[i][k] = 0.0f;
    if (live && r < dk) {
      if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(state + (long long)r * dv);
        S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
      } else {
        S[i][0] = state[(long long)r * dv];
      }
    }
  }
  const float const_e = p.decay ? p.decay[2 * h + 1] : 0.0f;
  pdl_wait();
  pdl_launch_dependents();
  for (int t = 0; t < p.S; ++t) {
    const long long row = (long long)b * p.S + t;
    const T* src = static_cast<const T*>(p.p) + row * p.ld;
    float v[V];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      v[k] = live ? to_f32(src[p.ov + h * dv + c0 + k]) : 0.0f;
      if (p.silu) v[k] = silu_f(v[k]);
    }
    for (int c = threadIdx.x; c < dk; c += kStepThreads) {
      float q = to_f32(src[p.oq + h * dk + c]), k = to_f32(src[p.ok + h * dk + c]);
      if (p.silu) {
        q = silu_f(q);
        k = silu_f(k);
      }
      qs[c] = q * p.q_scale;
      ks[c] = k;
      es[c] = p.decay ? const_e : expm1f(low_rank_log_decay<T>(p, row, h * dk + c));
    }
    __syncthreads();
    float acc[V];
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = 0.0f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = rg + kStepRows * i;
      if (r < dk) {
        const float e = es[r], kk = ks[r], q = qs[r];
#pragma unroll
        for (int k = 0; k < V; ++k) {
          S[i][k] += fmaf(e, S[i][k], kk * v[k]);
          acc[k] = fmaf(q, S[i][k], acc[k]);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k) {
      acc[k] += __shfl_xor_sync(0xffffffffu, acc[k], 16);
      if (lane < 16) red[warp * (kStepCols * V) + cg * V + k] = acc[k];
    }
    __syncthreads();
    const int out = threadIdx.x;
    if (out < kStepCols * V && blockIdx.x * kStepCols * V + out < dv) {
      float s = 0.0f;
#pragma unroll
      for (int w = 0; w < kStepThreads / 32; ++w) s += red[w * (kStepCols * V) + out];
      static_cast<T*>(p.o)[row * p.H * dv + (long long)h * dv + blockIdx.x * kStepCols * V + out] = from_f32<T>(s);
    }
  }
  if (!live) return;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = rg + kStepRows * i;
    if (r < dk) {
      if constexpr (V == 4)
        *reinterpret_cast<float4*>(state + (long long)r * dv) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
      else
        state[(long long)r * dv] = S[i][0];
    }
  }
}

// ------------------------------------------------------------------------------------------- decays of a long input
constexpr int kLinC = 64;           // tokens of a block
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float lin_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// log sigmoid(z) with its relative precision also where it is next to 0: log(1 + x) = 2 atanh(x / (2 + x)) by its odd series
// (x <= 1, so the argument is at most 1/3 and the first term left out is below 2 * 3^-13 / 13).
__device__ __forceinline__ float log_sigmoid_series_f(float z) {
  const float x = lin_exp2(-fabsf(z) * kLog2e);
  float s;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(s) : "f"(2.0f + x));
  s *= x;
  const float s2 = s * s;
  float r = 2.0f / 11;
  r = fmaf(r, s2, 2.0f / 9);
  r = fmaf(r, s2, 2.0f / 7);
  r = fmaf(r, s2, 2.0f / 5);
  r = fmaf(r, s2, 2.0f / 3);
  r = fmaf(r, s2, 2.0f);
  return fmaf(-r, s, fminf(z, 0.0f));
}

// A thread per key channel and block of 64 tokens.
template <typename T>
__global__ void __launch_bounds__(128) decay_kernel(const LinearParams p) {
  extern __shared__ float decay_r[];      // [rank][kLinC]
  constexpr int kHalf = kLinC / 2;
  const int t0 = blockIdx.x * kLinC, n = min(kLinC, p.S - t0), HK = p.H * p.dk;
  const long long row0 = (long long)blockIdx.z * p.S + t0;
  const int c = blockIdx.y * 128 + threadIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < kLinC * p.rank; i += 128) {
    const int t = i % kLinC, r = i / kLinC;
    decay_r[i] = t < n ? to_f32(static_cast<const T*>(p.p)[(row0 + t) * p.ld + p.orank + r]) : 0.0f;
  }
  __syncthreads();
  if (c >= HK) return;
  const float b = to_f32(static_cast<const T*>(p.b2)[c]), scale = p.inv_tau * kLog2e;
  const T* w = static_cast<const T*>(p.w2) + (long long)c * p.rank;
  float* out = p.log_a + row0 * HK + c;
  float G = 0.0f;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    f32x2 z[kHalf / 2];
#pragma unroll
    for (int t = 0; t < kHalf / 2; ++t) z[t] = f2_splat(b);
#pragma unroll 4
    for (int r = 0; r < p.rank; ++r) {
      const f32x2 wr = f2_splat(to_f32(w[r]));
#pragma unroll
      for (int t = 0; t < kHalf / 2; t += 2) {
        const float4 f = *reinterpret_cast<const float4*>(decay_r + r * kLinC + half * kHalf + 2 * t);
        z[t] = f2_fma(wr, f2_pack(f.x, f.y), z[t]);
        z[t + 1] = f2_fma(wr, f2_pack(f.z, f.w), z[t + 1]);
      }
    }
#pragma unroll
    for (int t = 0; t < kHalf; ++t) {
      float lo, hi;
      f2_unpack(z[t / 2], lo, hi);
      G += log_sigmoid_series_f(t & 1 ? hi : lo) * scale;
      if (half * kHalf + t < n) out[(long long)(half * kHalf + t) * HK] = G;
    }
  }
}

// ------------------------------------------------------------------------------------------- pieces of 64 tokens
constexpr int kLinThreads = 4;      // threads per value column of a CTA
constexpr float kLinSpan = 72.0f;   // log2 decay span of a piece
constexpr int kPRow = kLinC + 8;    // padded rows (of the scores): ldmatrix without bank conflicts

__device__ __forceinline__ void lin_ldm(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lin_ldm_t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lin_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 f = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - f.x, b - f.y);
}

__device__ __forceinline__ void lin_cp16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void lin_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void lin_cp_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// STAGED: the rows of the next piece (queries, keys, log decays) are copied to shared memory while this one is multiplied;
// with 256 key channels there is no room for that.
template <int DK, int DV, bool OUT>
struct LinSmem {
  static constexpr bool kStaged = DK <= 128;
  static constexpr int kThreads = kLinThreads * DV;
  static constexpr int kKRow = DK + 8;
  static constexpr int kVRow = DV + 8;
  static constexpr int kPBytes = kLinC * kPRow * 2;
  static constexpr int kKBytes = kLinC * kKRow * 2;       // one part of the keys (or queries)
  static constexpr int kVBytes = kLinC * kVRow * 2;
  static constexpr int kSBytes = DK * kVRow * 2;
  static constexpr int kK = 0;                            // [2][64][DK + 8] high, low; if not STAGED the scores take its place
  static constexpr int kV = kK + 2 * kKBytes;
  static constexpr int kQ = kV + (kStaged ? 2 : 1) * kVBytes;   // pass 2 only from here
  static constexpr int kS = kQ + (OUT ? 2 * kKBytes : 0);
  static constexpr int kGate = kS + (OUT ? 2 * kSBytes : 0);
  static constexpr int kParts = 2 * kThreads / DK;     // a thread prepares two channels of 64 / kParts tokens
  static constexpr int kRawK = kGate + 2 * DK * 4;
  static constexpr int kRawQ = kRawK + (kStaged ? kLinC * DK * 2 : 0);
  static constexpr int kRawA = kRawQ + (kStaged && OUT ? kLinC * DK * 2 : 0);
  static constexpr int kP = kStaged ? kRawA + kLinC * DK * 4 : kK;   // scores, [2][64][64 + 8]
  static constexpr int kTotal = kStaged ? kP + (OUT ? 2 * kPBytes : 0) : kRawA;
  static_assert(kStaged || kPBytes <= kKBytes, "the scores fit where the keys were");
  static_assert(kTotal <= 227 * 1024, "linear attention: shared memory budget");
};

// One CTA: DV value columns of one head over one segment.  OUT = false: the segment's contribution to the state (pass 1).
template <int DK, int DV, bool OUT>
__global__ void __launch_bounds__(kLinThreads * DV, DK <= 64 && DV <= 64 ? 2 : 1) linear_chunk_kernel(const LinearParams p) {
  using L = LinSmem<DK, DV, OUT>;
  using bf = __nv_bfloat16;
  constexpr bool STAGED = L::kStaged;
  constexpr int KR = L::kKRow, kVRow = L::kVRow, NTHR = L::kThreads;
  constexpr int WARPS = NTHR / 32;
  constexpr int MT = DK / 16;                     // 16-row tiles of the state
  constexpr int MTW = MT > WARPS ? MT / WARPS : 1;        // ... of a warp
  constexpr int WN = MT < WARPS ? WARPS / MT : 1; // warps side by side along the columns
  constexpr int NT = DV / 8 / WN;                 // 8-column tiles of a warp
  constexpr int NA = 4 * 64 / 8 / WARPS;          // 8-column tiles of a warp's scores (64 x 64 over all warps)
  static_assert(NT % 2 == 0 && NA % 2 == 0, "fragments of B come in pairs");
  constexpr int TP = kLinC / L::kParts;           // tokens a thread prepares
  extern __shared__ __align__(16) uint8_t lin_smem[];
  bf* kh = reinterpret_cast<bf*>(lin_smem + L::kK);
  bf* kl = kh + kLinC * KR;
  bf* vs = reinterpret_cast<bf*>(lin_smem + L::kV);
  bf* qh = reinterpret_cast<bf*>(lin_smem + L::kQ);
  bf* ql = qh + kLinC * KR;
  bf* sh = reinterpret_cast<bf*>(lin_smem + L::kS);
  bf* sl = sh + DK * kVRow;
  bf* ph = reinterpret_cast<bf*>(lin_smem + L::kP);
  bf* pl = ph + kLinC * kPRow;
  float* g_in = reinterpret_cast<float*>(lin_smem + L::kGate);  // factor on the state before the piece's products
  float* g_out = g_in + DK;                       // ... and after them
  bf* raw_k = reinterpret_cast<bf*>(lin_smem + L::kRawK);       // [64][DK]
  bf* raw_q = reinterpret_cast<bf*>(lin_smem + L::kRawQ);
  float* raw_a = reinterpret_cast<float*>(lin_smem + L::kRawA);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seg = blockIdx.x, b = blockIdx.z;
  const int vt = (p.dv + DV - 1) / DV;
  const int h = blockIdx.y / vt, v0 = (blockIdx.y % vt) * DV;
  const int dk = p.dk, dv = p.dv, HK = p.H * dk;
  const int t_begin = seg * p.seg_tokens, t_end = min(p.S, t_begin + p.seg_tokens);
  const long long row_b = (long long)b * p.S;
  const bf* rows = static_cast<const bf*>(p.p) + row_b * p.ld;
  const float* la_base = p.log_a ? p.log_a + row_b * HK + h * dk : nullptr;
  pdl_wait();
  pdl_launch_dependents();
  const float const_la = p.decay ? p.decay[2 * h] * kLog2e : 0.0f;
  const float q_shift = OUT ? log2f(p.q_scale) : 0.0f;
  const int ch = tid % (DK / 2) * 2, part = tid / (DK / 2);   // this thread's channels and share of the tokens while preparing

  // Values of the piece at t0 into buffer `buf`; with STAGED everything else of it too.
  auto fetch = [&](int t0, int buf) {
    bf* v = vs + buf * (kLinC * kVRow);
    for (int i = tid; i < kLinC * DV / 8; i += NTHR) {
      const int t = i / (DV / 8), c = i % (DV / 8) * 8;
      const bool ok = t0 + t < t_end && v0 + c < dv;
      lin_cp16(v + t * kVRow + c, ok ? rows + (long long)(t0 + t) * p.ld + p.ov + h * dv + v0 + c : rows, ok);
    }
    if constexpr (STAGED) {
      for (int i = tid; i < kLinC * DK / 8; i += NTHR) {
        const int t = i / (DK / 8), c = i % (DK / 8) * 8;
        const bool ok = t0 + t < t_end && c < dk;
        const bf* r = ok ? rows + (long long)(t0 + t) * p.ld + h * dk + c : rows;
        lin_cp16(raw_k + t * DK + c, ok ? r + p.ok : r, ok);
        if (OUT) lin_cp16(raw_q + t * DK + c, ok ? r + p.oq : r, ok);
      }
      if (la_base) {
        for (int i = tid; i < kLinC * DK / 4; i += NTHR) {
          const int t = i / (DK / 4), c = i % (DK / 4) * 4;
          const bool ok = t0 + t < t_end && c < dk;
          lin_cp16(raw_a + t * DK + c, ok ? la_base + (long long)(t0 + t) * HK + c : la_base, ok);
        }
      }
    }
    lin_cp_commit();
  };
  // Token t of the piece at t0, channels ch and ch + 1 (channels beyond dk are zero): the decay summed from the block's start
  // (constant decays: from the piece's).
  auto decayed = [&](int t0, int t) -> float2 {
    if (!la_base) return make_float2((t + 1) * const_la, (t + 1) * const_la);
    if constexpr (STAGED) return *reinterpret_cast<const float2*>(raw_a + t * DK + ch);
    return ch < dk ? *reinterpret_cast<const float2*>(la_base + (long long)(t0 + t) * HK + ch) : make_float2(0.0f, 0.0f);
  };
  auto pair_of = [&](const bf* raw, int col, int t0, int t) -> float2 {
    if constexpr (STAGED) return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(raw + t * DK + ch));
    if (ch >= dk) return make_float2(0.0f, 0.0f);
    return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(rows + (long long)(t0 + t) * p.ld + col + h * dk + ch));
  };

  // the state: warp's row tiles m0 + 128 * i and column tiles n0 + 8 * j
  const int m0 = (warp / WN) * 16, n0 = (warp % WN) * NT * 8;
  float S[MTW][NT][4];
  auto for_state = [&](auto f) {
#pragma unroll
    for (int i = 0; i < MTW; ++i)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; e += 2)
          f(i, j, e, m0 + i * 16 * WARPS + (lane >> 2) + (e >> 1) * 8, n0 + j * 8 + (lane & 3) * 2);
  };
  const long long mat = (long long)dk * dv, bh = (long long)b * p.H + h;
  float* ends = p.ends + bh * (p.segments + 1) * mat;
  float* totals = p.totals + bh * p.segments * dk;
  for_state([&](int i, int j, int e, int r, int c) {
    S[i][j][e] = S[i][j][e + 1] = 0.0f;
    if ((OUT || seg == 0) && r < dk && v0 + c < dv) {
      // pass 1 starts the first segment from the state itself and leaves a copy: pass 2 replaces the state
      const float* src = (OUT && p.segments > 1 ? ends + p.segments * mat : p.state + bh * mat) + (long long)r * dv + v0 + c;
      const float2 f = *reinterpret_cast<const float2*>(src);
      S[i][j][e] = f.x;
      S[i][j][e + 1] = f.y;
      if (!OUT) *reinterpret_cast<float2*>(ends + p.segments * mat + (long long)r * dv + v0 + c) = f;
    }
  });
  if (OUT && seg > 0) {
    for_state([&](int i, int j, int e, int r, int c) {
      if (r < dk && v0 + c < dv) {
        float2 s = *reinterpret_cast<const float2*>(ends + (long long)r * dv + v0 + c);
#pragma unroll 4
        for (int k = 1; k < seg; ++k) {
          const float2 f = *reinterpret_cast<const float2*>(ends + k * mat + (long long)r * dv + v0 + c);
          const float d = totals[k * dk + r];
          s.x += fmaf(d, s.x, f.x);
          s.y += fmaf(d, s.y, f.y);
        }
        S[i][j][e] = s.x;
        S[i][j][e + 1] = s.y;
      }
    });
  }
  float2 total = make_float2(0.0f, 0.0f);         // of this thread's channels (threads with part == 0)
  float2 base = make_float2(0.0f, 0.0f);          // decay of the block before the piece
  int buf = 0;
  // A fetch has arrived: this thread's copies of the values pass through their activation, in place.
  auto arrived = [&](int buf) {
    lin_cp_wait();
    if (p.silu) {
      for (int i = tid; i < kLinC * DV / 8; i += NTHR) {
        uint4* at = reinterpret_cast<uint4*>(vs + buf * (kLinC * kVRow) + i / (DV / 8) * kVRow + i % (DV / 8) * 8);
        uint4 u = *at;
        uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float2 f = unpack_bf16x2(w[k]);
          w[k] = pack_bf16x2(fast_silu_f(f.x), fast_silu_f(f.y));
        }
        *at = u;
      }
    }
  };
  if (t_begin < t_end) fetch(t_begin, 0);
  arrived(0);
  __syncthreads();
  // Three barriers a piece in pass 2: everyone is done with the one before (and agrees on this one's length); operands are
  // there; scores and the next piece's rows are there.  Two in pass 1: rows are there; operands are there.
  for (int t0 = t_begin; t0 < t_end;) {
    int n = min(kLinC - t0 % kLinC, t_end - t0);  // pieces do not cross blocks
    const bf* v_now = vs + buf * (kLinC * kVRow);
    // ---- a piece whose decays span too much becomes shorter
    auto decay_to = [&](int t) {
      float2 g = decayed(t0, t);
      if (la_base) {
        g.x -= base.x;
        g.y -= base.y;
      }
      return g;
    };
    if (!OUT) __syncthreads();
    float2 all = decay_to(n - 1), first = make_float2(0.0f, 0.0f);
    if constexpr (OUT) {
      first = decay_to(0);
      while (__syncthreads_or(fminf(all.x - first.x, all.y - first.y) < -kLinSpan) && n > 1) {
        n = (n + 3) / 4;
        all = decay_to(n - 1);
      }
    }
    if (part == 0) {
      *reinterpret_cast<float2*>(g_in + ch) = OUT ? make_float2(lin_exp2(first.x), lin_exp2(first.y)) :
                                                    make_float2(lin_exp2(all.x), lin_exp2(all.y));
      *reinterpret_cast<float2*>(g_out + ch) = make_float2(lin_exp2(all.x - first.x), lin_exp2(all.y - first.y));
      total.x += all.x;
      total.y += all.y;
    }
    // ---- operands: k e^{G_1 - G_j} and q e^{G_i - G_1}; pass 1: k e^{G_end - G_j}
    const float2 ref = OUT ? first : all, ref_q = make_float2(first.x - q_shift, first.y - q_shift);
#pragma unroll
    for (int i = 0; i < TP; ++i) {
      const int t = part * TP + i;
      float2 k = make_float2(0.0f, 0.0f), q = k;
      if (t < n) {
        const float2 G = decay_to(t);
        k = pair_of(raw_k, p.ok, t0, t);
        if (p.silu) k = unpack_bf16x2(pack_bf16x2(fast_silu_f(k.x), fast_silu_f(k.y)));
        k.x *= lin_exp2(ref.x - G.x);
        k.y *= lin_exp2(ref.y - G.y);
        if (OUT) {
          q = pair_of(raw_q, p.oq, t0, t);
          if (p.silu) q = make_float2(fast_silu_f(q.x), fast_silu_f(q.y));
          q.x *= lin_exp2(G.x - ref_q.x);
          q.y *= lin_exp2(G.y - ref_q.y);
        }
      }
      uint32_t hi, lo;
      split_pair(k.x, k.y, hi, lo);
      *reinterpret_cast<uint32_t*>(kh + t * KR + ch) = hi;
      *reinterpret_cast<uint32_t*>(kl + t * KR + ch) = lo;
      if (OUT) {
        split_pair(q.x, q.y, hi, lo);
        *reinterpret_cast<uint32_t*>(qh + t * KR + ch) = hi;
        *reinterpret_cast<uint32_t*>(ql + t * KR + ch) = lo;
      }
    }
    __syncthreads();
    if (STAGED && t0 + n < t_end) fetch(t0 + n, buf ^ 1);
    // ---- the state as the piece's first token sees it
    for_state([&](int i, int j, int e, int r, int c) {
      const float g = g_in[r];
      S[i][j][e] *= g;
      S[i][j][e + 1] *= g;
      if (OUT) {
        uint32_t hi, lo;
        split_pair(S[i][j][e], S[i][j][e + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(sh + r * kVRow + c) = hi;
        *reinterpret_cast<uint32_t*>(sl + r * kVRow + c) = lo;
      }
    });
    // this warp's 16 x 32 part of the outputs; the row tiles, whose causal work differs, rotate over the schedulers
    const int mt = (warp + (warp >> 2)) & 3, nh = (warp >> 2) * 32;
    const int a_row = lane & 15, a_col = (lane >> 4) * 8;                          // fragments of A, row-major
    const int b_row = (lane & 7) + ((lane >> 4) & 1) * 8, b_col = ((lane >> 3) & 1) * 8;   // of B stored [n][k]
    const int bt_row = (lane & 7) + ((lane >> 3) & 1) * 8, bt_col = ((lane >> 4) & 1) * 8; // of B stored [k][n]
    const int na = (warp >> 2) * NA * 8;                  // ... and its 16 x 8 NA part of the scores
    float a[NA][4];
    if constexpr (OUT) {
      // ---- scores of the piece's own tokens
#pragma unroll
      for (int j = 0; j < NA; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) a[j][e] = 0.0f;
      if (na <= mt * 16 + 15) {
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          uint32_t ah[4], al[4];
          lin_ldm(ah, qh + (mt * 16 + a_row) * KR + kk * 16 + a_col);
          lin_ldm(al, ql + (mt * 16 + a_row) * KR + kk * 16 + a_col);
          uint32_t bh4[NA / 2][4], bl4[NA / 2][4];
#pragma unroll
          for (int j = 0; j < NA / 2; ++j) {
            lin_ldm(bh4[j], kh + (na + j * 16 + b_row) * KR + kk * 16 + b_col);
            lin_ldm(bl4[j], kl + (na + j * 16 + b_row) * KR + kk * 16 + b_col);
          }
          // neighbouring products go to different accumulators
#pragma unroll
          for (int j = 0; j < NA; ++j) lin_mma(a[j], ah, bh4[j / 2][j % 2 * 2], bh4[j / 2][j % 2 * 2 + 1]);
#pragma unroll
          for (int j = 0; j < NA; ++j) lin_mma(a[j], ah, bl4[j / 2][j % 2 * 2], bl4[j / 2][j % 2 * 2 + 1]);
#pragma unroll
          for (int j = 0; j < NA; ++j) lin_mma(a[j], al, bh4[j / 2][j % 2 * 2], bh4[j / 2][j % 2 * 2 + 1]);
        }
      }
    }
    auto put_scores = [&]() {
#pragma unroll
      for (int j = 0; j < NA; ++j)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int r = mt * 16 + (lane >> 2) + (e >> 1) * 8, c = na + j * 8 + (lane & 3) * 2;
          uint32_t hi, lo;
          split_pair(c <= r ? a[j][e] : 0.0f, c + 1 <= r ? a[j][e + 1] : 0.0f, hi, lo);
          *reinterpret_cast<uint32_t*>(ph + r * kPRow + c) = hi;
          *reinterpret_cast<uint32_t*>(pl + r * kPRow + c) = lo;
        }
    };
    if (OUT && STAGED) put_scores();
    // ---- the state after the piece
#pragma unroll
    for (int kk = 0; kk < kLinC / 16; ++kk) {
      uint32_t vb[NT / 2][4];
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) lin_ldm_t(vb[j], v_now + (kk * 16 + bt_row) * kVRow + n0 + j * 16 + bt_col);
#pragma unroll
      for (int i = 0; i < MTW; ++i) {
        uint32_t ah[4], al[4];      // transposed: rows are key channels
        lin_ldm_t(ah, kh + (kk * 16 + b_row) * KR + m0 + i * 16 * WARPS + b_col);
        lin_ldm_t(al, kl + (kk * 16 + b_row) * KR + m0 + i * 16 * WARPS + b_col);
#pragma unroll
        for (int j = 0; j < NT; ++j) lin_mma(S[i][j], ah, vb[j / 2][(j & 1) * 2], vb[j / 2][(j & 1) * 2 + 1]);
#pragma unroll
        for (int j = 0; j < NT; ++j) lin_mma(S[i][j], al, vb[j / 2][(j & 1) * 2], vb[j / 2][(j & 1) * 2 + 1]);
      }
    }
    if constexpr (OUT) {
      for_state([&](int i, int j, int e, int r, int c) {
        const float g = g_out[r];
        S[i][j][e] *= g;
        S[i][j][e + 1] *= g;
      });
      if (!STAGED) {
        __syncthreads();        // the keys are done with: the scores take their place
        put_scores();
      }
      if (STAGED && t0 + n < t_end) arrived(buf ^ 1);
      __syncthreads();
      // ---- outputs: own tokens, then everything before the piece
      float o[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.0f;
      for (int kk = 0; kk <= mt; ++kk) {
        uint32_t ah[4], al[4];
        lin_ldm(ah, ph + (mt * 16 + a_row) * kPRow + kk * 16 + a_col);
        lin_ldm(al, pl + (mt * 16 + a_row) * kPRow + kk * 16 + a_col);
        uint32_t vb[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) lin_ldm_t(vb[j], v_now + (kk * 16 + bt_row) * kVRow + nh + j * 16 + bt_col);
#pragma unroll
        for (int j = 0; j < 4; ++j) lin_mma(o[j], ah, vb[j / 2][j % 2 * 2], vb[j / 2][j % 2 * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 4; ++j) lin_mma(o[j], al, vb[j / 2][j % 2 * 2], vb[j / 2][j % 2 * 2 + 1]);
      }
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t ah[4], al[4];
        lin_ldm(ah, qh + (mt * 16 + a_row) * KR + kk * 16 + a_col);
        lin_ldm(al, ql + (mt * 16 + a_row) * KR + kk * 16 + a_col);
        uint32_t bh4[2][4], bl4[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          lin_ldm_t(bh4[j], sh + (kk * 16 + bt_row) * kVRow + nh + j * 16 + bt_col);
          lin_ldm_t(bl4[j], sl + (kk * 16 + bt_row) * kVRow + nh + j * 16 + bt_col);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) lin_mma(o[j], ah, bh4[j / 2][j % 2 * 2], bh4[j / 2][j % 2 * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 4; ++j) lin_mma(o[j], ah, bl4[j / 2][j % 2 * 2], bl4[j / 2][j % 2 * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 4; ++j) lin_mma(o[j], al, bh4[j / 2][j % 2 * 2], bh4[j / 2][j % 2 * 2 + 1]);
      }
      bf* out = static_cast<bf*>(p.o) + (row_b + t0) * p.H * dv + (long long)h * dv + v0;
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int r = mt * 16 + (lane >> 2) + (e >> 1) * 8, c = nh + j * 8 + (lane & 3) * 2;
          if (r < n && v0 + c < dv)
            *reinterpret_cast<uint32_t*>(out + (long long)r * p.H * dv + c) = pack_bf16x2(o[j][e], o[j][e + 1]);
        }
    }
    t0 += n;
    base = t0 % kLinC ? make_float2(base.x + all.x, base.y + all.y) : make_float2(0.0f, 0.0f);
    if (STAGED) {
      if (!OUT && t0 < t_end) arrived(buf ^ 1);
      buf ^= 1;
    } else if (t0 < t_end) {
      __syncthreads();
      fetch(t0, 0);
      arrived(0);
      __syncthreads();
    }
  }
  if (OUT && seg != p.segments - 1) return;
  float* dst = OUT ? p.state + bh * mat : ends + seg * mat;
  for_state([&](int i, int j, int e, int r, int c) {
    if (r < dk && v0 + c < dv)
      *reinterpret_cast<float2*>(dst + (long long)r * dv + v0 + c) = make_float2(S[i][j][e], S[i][j][e + 1]);
  });
  if (!OUT && v0 == 0 && part == 0 && ch < dk) *reinterpret_cast<float2*>(totals + seg * dk + ch) =
        make_float2(expm1f(total.x * 0.6931471805599453f), expm1f(total.y * 0.6931471805599453f));
}

// ------------------------------------------------------------------------------------------- norm and gate
struct HeadNormParams {
  const void* o;            // [rows, groups * n]
  const void* w;            // [n]
  const void* g;            // [rows, ldg], same columns as o
  long long ldg;
  void* out;                // [rows, groups * n]
  int groups, n, sigmoid;
  float eps;
};

// LG lanes per (row, group); 128: a whole CTA.
template <typename T, int V, int LG>
__global__ void __launch_bounds__(128) head_norm_gate_kernel(const HeadNormParams p, int units) {
  __shared__ float scratch[33];
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int kKeep = LG == 128 ? 4 : 2;
  const int lane = threadIdx.x % LG;
  const int wanted = blockIdx.x * (128 / LG) + threadIdx.x / LG, unit = min(wanted, units - 1);
  pdl_wait();
  pdl_launch_dependents();
  const int row = unit / p.groups, off = (unit - row * p.groups) * p.n;
  const long long at = (long long)row * p.groups * p.n + off;
  const T* o = static_cast<const T*>(p.o) + at;
  const T* g = static_cast<const T*>(p.g) + row * p.ldg + off;
  T* out = static_cast<T*>(p.out) + at;
  auto load = [&](const T* q, float (&x)[V]) {
    if constexpr (V == 8) Vec8<T>::load(q, x);
    else x[0] = to_f32(q[0]);
  };
  float keep[kKeep][V], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (i * LG + lane) * V;
#pragma unroll
    for (int k = 0; k < V; ++k) keep[i][k] = 0.0f;
    if (c < p.n) load(o + c, keep[i]);
  }
#pragma unroll
  for (int i = 0; i < kKeep; ++i)
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(keep[i][k], keep[i][k], ss);
  for (int c = (kKeep * LG + lane) * V; c < p.n; c += LG * V) {
    float x[V];
    load(o + c, x);
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(x[k], x[k], ss);
  }
  if constexpr (LG == 128) {
    ss = block_sum(ss, scratch);
  } else {
#pragma unroll
    for (int x = LG / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
  }
  const float inv = 1.0f / sqrtf(ss / (float)p.n + p.eps);
  if (wanted >= units) return;
  auto put = [&](int c, const float (&x)[V]) {
    float w[V], gv[V], y[V];
    load(static_cast<const T*>(p.w) + c, w);
    load(g + c, gv);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float s = FAST ? __fdividef(1.0f, 1.0f + __expf(-gv[k])) : 1.0f / (1.0f + expf(-gv[k]));
      y[k] = x[k] * inv * w[k] * (p.sigmoid ? s : gv[k] * s);
    }
    if constexpr (V == 8) Vec8<T>::store(out + c, y);
    else out[c] = from_f32<T>(y[0]);
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (i * LG + lane) * V;
    if (c < p.n) put(c, keep[i]);
  }
  for (int c = (kKeep * LG + lane) * V; c < p.n; c += LG * V) {
    float x[V];
    load(o + c, x);
    put(c, x);
  }
}
template <typename T, int V>
static int launch_head_norm(const HeadNormParams& p, int units, cudaStream_t st) {
  const int vecs = (p.n + V - 1) / V;
#define DPTB_HN(LG) return counted(1, (int)launch_k(head_norm_gate_kernel<T, V, LG>, dim3((units + 128 / LG - 1) / (128 / LG)), \
                                                    dim3(128), (size_t)0, st, p, units))
  if (vecs <= 8) DPTB_HN(8);
  if (vecs <= 16) DPTB_HN(16);
  if (vecs <= 96) DPTB_HN(32);
  DPTB_HN(128);
#undef DPTB_HN
}

template <typename T, int V>
static int launch_step(const LinearParams& p, cudaStream_t st) {
  const dim3 grid((p.dv + kStepCols * V - 1) / (kStepCols * V), p.H, p.B);
  const size_t smem = (3 * p.dk + 8 * kStepCols * V) * sizeof(float);
  const int nr = (p.dk + kStepRows - 1) / kStepRows;
#define DPTB_STEP(NRV) return counted(1, (int)launch_k(linear_step_kernel<T, V, NRV>, grid, dim3(kStepThreads), smem, st, p))
  if (nr <= 2) DPTB_STEP(2);
  if (nr <= 4) DPTB_STEP(4);
  if (nr <= 8) DPTB_STEP(8);
  if (nr <= 16) DPTB_STEP(16);
  if (nr <= 32) DPTB_STEP(32);
#undef DPTB_STEP
  return kErrUnsupported;
}

template <int DK, int DV>
static int launch_chunks(const LinearParams& p, cudaStream_t st) {
  using L1 = LinSmem<DK, DV, false>;
  using L2 = LinSmem<DK, DV, true>;
  static bool configured = false;
  if (!configured) {
    DPTB_CUDA_OK(cudaFuncSetAttribute(linear_chunk_kernel<DK, DV, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, L1::kTotal));
    DPTB_CUDA_OK(cudaFuncSetAttribute(linear_chunk_kernel<DK, DV, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, L2::kTotal));
    configured = true;
  }
  const unsigned gy = p.H * ((p.dv + DV - 1) / DV);
  if (p.segments > 1) {
    const int rc = counted(1, (int)launch_k(linear_chunk_kernel<DK, DV, false>, dim3(p.segments - 1, gy, p.B), dim3(L1::kThreads),
                                            (size_t)L1::kTotal, st, p));
    if (rc) return rc;
  }
  return counted(1, (int)launch_k(linear_chunk_kernel<DK, DV, true>, dim3(p.segments, gy, p.B), dim3(L2::kThreads),
                                  (size_t)L2::kTotal, st, p));
}

}  // namespace dptb

using namespace dptb;

struct DptbLinearArgs {
  const void* p; const void* w2; const void* b2; const float* decay; float* log_a; float* state; void* o; float* ws;
  long long ld, ws_floats;
  int oq, ok, ov, orank;
  int B, S, H, dk, dv, rank, silu, f32, chunked, segments;
  float q_scale, inv_tau;
};

// Whether long inputs of these sizes run as pieces on the tensor cores.
extern "C" int dptb_linear_chunkable(int dk, int dv, int f32) { return !f32 && dk <= 256 && dk % 8 == 0 && dv % 8 == 0; }

static int linear_seg_tokens(int S, int segments) { return ((S + segments - 1) / segments + kLinC - 1) / kLinC * kLinC; }

// Value columns of a CTA.
static int linear_dv(int dk, int dv) { return dk <= 64 && dv > 64 ? 128 : 64; }

// Segments: as many CTAs as run at once (two of 64 columns fit an SM up to 64 key channels), four pieces each at least.
extern "C" int dptb_linear_segments(int B, int S, int H, int dk, int dv) {
  const int cols = linear_dv(dk, dv), ctas = B * H * ((dv + cols - 1) / cols);
  int s = sm_count() * (dk <= 64 && cols == 64 ? 2 : 1) / ctas;
  const int by_len = S / (4 * kLinC);
  if (s > by_len) s = by_len;
  if (s < 1) s = 1;
  const int seg = linear_seg_tokens(S, s);
  return (S + seg - 1) / seg;
}
extern "C" long long dptb_linear_ws_floats(int B, int H, int dk, int dv, int segments) {
  return segments <= 1 ? 0 : (long long)B * H * ((long long)(segments + 1) * dk * dv + (long long)segments * dk);
}

extern "C" int dptb_linear_attn(const DptbLinearArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->B <= 0 || a->S <= 0) return 0;
  if (a->H <= 0 || a->dk <= 0 || a->dv <= 0 || a->B > 65535 || a->H > 65535) return kErrBadShape;
  if (!a->decay && (!a->w2 || !a->b2 || a->rank <= 0)) return kErrBadShape;
  LinearParams p = {};
  p.p = a->p; p.ld = a->ld; p.oq = a->oq; p.ok = a->ok; p.ov = a->ov; p.orank = a->orank;
  p.w2 = a->w2; p.b2 = a->b2; p.decay = a->decay; p.state = a->state; p.o = a->o;
  p.B = a->B; p.S = a->S; p.H = a->H; p.dk = a->dk; p.dv = a->dv; p.rank = a->rank; p.silu = a->silu;
  p.q_scale = a->q_scale; p.inv_tau = a->inv_tau;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (!a->chunked) {
    p.segments = 1;
    p.seg_tokens = a->S;
    if (a->dv % 4 == 0 && al16(a->state)) return a->f32 ? launch_step<float, 4>(p, st) : launch_step<__nv_bfloat16, 4>(p, st);
    return a->f32 ? launch_step<float, 1>(p, st) : launch_step<__nv_bfloat16, 1>(p, st);
  }
  if (!dptb_linear_chunkable(a->dk, a->dv, a->f32) || a->q_scale <= 0.0f) return kErrUnsupported;
  if (a->ld % 8 || a->oq % 8 || a->ok % 8 || a->ov % 8 || !al16(a->log_a) || !al16(a->p) || !al16(a->state) || !al16(a->o)) return kErrBadShape;
  p.segments = a->segments < 1 ? 1 : a->segments;
  p.seg_tokens = linear_seg_tokens(a->S, p.segments);
  if ((a->S + p.seg_tokens - 1) / p.seg_tokens != p.segments) return kErrBadShape;
  if (dptb_linear_ws_floats(a->B, a->H, a->dk, a->dv, p.segments) > a->ws_floats) return kErrTooLarge;
  if (p.segments > 1 && !al16(a->ws)) return kErrBadShape;
  p.ends = a->ws;
  p.totals = a->ws ? a->ws + (long long)a->B * a->H * (p.segments + 1) * a->dk * a->dv : nullptr;
  if (!a->decay) {
    if (!a->log_a) return kErrBadShape;
    p.log_a = a->log_a;
    const size_t smem = (size_t)kLinC * a->rank * sizeof(float);
    if (smem > 48 * 1024) return kErrTooLarge;
    const dim3 grid((a->S + kLinC - 1) / kLinC, (a->H * a->dk + 127) / 128, a->B);
    const int rc = counted(1, (int)launch_k(decay_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, p));
    if (rc) return rc;
  }
  const bool wide = linear_dv(a->dk, a->dv) == 128;
  if (a->dk <= 32) return wide ? launch_chunks<32, 128>(p, st) : launch_chunks<32, 64>(p, st);
  if (a->dk <= 64) return wide ? launch_chunks<64, 128>(p, st) : launch_chunks<64, 64>(p, st);
  if (a->dk <= 128) return launch_chunks<128, 64>(p, st);
  return launch_chunks<256, 64>(p, st);
}

struct DptbHeadNormArgs {
  const void* o; const void* w; const void* g; void* out;
  long long ldg;
  int rows, groups, n, sigmoid, f32;
  float eps;
};

extern "C" int dptb_head_norm_gate(const DptbHeadNormArgs* a, void* stream_v) {
  auto st = static_cast<cudaStream_t>(stream_v);
  if (a->rows <= 0) return 0;
  if (a->groups <= 0 || a->n <= 0 || a->ldg < (long long)a->groups * a->n) return kErrBadShape;
  HeadNormParams p;
  p.o = a->o; p.w = a->w; p.g = a->g; p.ldg = a->ldg; p.out = a->out;
  p.groups = a->groups; p.n = a->n; p.sigmoid = a->sigmoid; p.eps = a->eps;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = a->n % 8 == 0 && a->ldg % 8 == 0 && al16(a->o) && al16(a->w) && al16(a->g) && al16(a->out);
  const long long units = (long long)a->rows * a->groups;
  if (units > 0x7fffffff - 128) return kErrTooLarge;
  if (a->f32) return vec ? launch_head_norm<float, 8>(p, (int)units, st) : launch_head_norm<float, 1>(p, (int)units, st);
  return vec ? launch_head_norm<__nv_bfloat16, 8>(p, (int)units, st) : launch_head_norm<__nv_bfloat16, 1>(p, (int)units, st);
}
