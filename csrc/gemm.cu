// bf16 GEMM on 5th-generation tensor cores (tcgen05 + TMEM) with fused epilogues, plus a plain
// SIMT kernel for shapes / dtypes the tensor-core path cannot take.
//
//   C[M,N] = epilogue( op(A)[M,K] * op(B)[K,N] )
//
// It replaces the reference's single 32x32 shared-memory-tiled fp32 matmul and the transpose /
// row-broadcast-add / activation kernels around it (reference: lib/native/src/kernels/matmul.cuh:27-63,
// lib/native/src/kernels/transpose.cuh:12-29, lib/native/src/kernels/elementwise.cuh:64-73).
//
// Structure of the tensor-core kernel (one persistent CTA per SM, 320 threads):
//   warp 0      TMA producer: one elected lane streams 128xBK / BNxBK tiles into a STAGES-deep ring.
//   warp 1      MMA issuer: one elected lane issues tcgen05.mma (M=128, N=BN, K=16) into one of two
//               TMEM accumulators; tcgen05.commit releases smem stages and publishes accumulators.
//   warps 2-9   epilogue (two warps per TMEM lane quarter, alternating 64-column blocks): tcgen05.ld of the
//               finished accumulator (one row per thread), bias / activation / residual / accumulate in
//               registers, bf16 or fp32 stores, while the issuer already works on the next tile in the
//               other accumulator.
#include "gemm_tc.cuh"

namespace dptb {

// Registry of the per-translation-unit status blocks (filled by static initialisers at load time).
static int (*g_status_blocks[64])(int*, int);
static int g_num_status_blocks = 0;
void register_status_block(int (*access)(int*, int)) {
  if (g_num_status_blocks < 64) g_status_blocks[g_num_status_blocks++] = access;
}

// ----------------------------------------------------------------------------- SIMT fallback
// Any shape, any stride, fp32 or bf16 inputs.  64x64 tile, 16x16 threads, 4x4 outputs per thread.
template <typename TA, typename TB>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const TA* __restrict__ A, long long sam, long long sak, const TB* __restrict__ B, long long sbk,
                 long long sbn, const GemmParams p) {
  __shared__ float As[16][64 + 1];
  __shared__ float Bs[16][64 + 1];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const long long m0 = (long long)blockIdx.y * 64, n0 = (long long)blockIdx.x * 64;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
    for (int i = threadIdx.x; i < 16 * 64; i += 256) {
      const int kk = i & 15, mm = i >> 4;
      const long long m = m0 + mm, n = n0 + mm, k = k0 + kk;
      As[kk][mm] = (m < p.M && k < p.K) ? (float)A[m * sam + k * sak] : 0.0f;
      Bs[kk][mm] = (n < p.N && k < p.K) ? (float)B[k * sbk + n * sbn] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = Bs[kk][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 4; ++j) {
      const long long m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < p.M && n < p.N) epilogue_scalar(p, m, n, acc[i][j]);
    }
}

}  // namespace dptb

using namespace dptb;

// Peer-memory description of the all-gather prologue (see TpAg): every rank's shard of A, [rows_per_rank, lda] each.
struct DptbTpAgArgs {
  int world, rank;
  long long rows_per_rank;
  const void* a_peer[kMaxRanks];
  const void* ready;   // local flag words [kMaxRanks], raised by dptb_tp_signal on the peers
  const void* epoch;   // local word written by this rank's dptb_tp_signal: the value the flags must have reached
};
// 32-bit words of a flag array for `max_tiles` tiles.
extern "C" long long dptb_tp_flag_words(int max_tiles) { return ((long long)max_tiles + 1) * kMaxRanks; }

static int gemm_impl(const DptbGemmArgs* a, const DptbTpArArgs* ar, const DptbTpAgArgs* ag, void* stream_v) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_v);
  if (a->M <= 0 || a->N <= 0) return 0;
  if (a->K < 0) return kErrBadShape;
  GemmParams p;
  p.ar.world = 0;
  p.ar.mode = 0;
  p.ar.rows_per_rank = 0;
  p.ag.world = 0;
  const void* a_ptr = a->A;
  if (ag) {
    if (ar || ag->world < 1 || ag->world > kMaxRanks || ag->rank < 0 || ag->rank >= ag->world) return kErrBadShape;
    if (a->trans_a || !a->trans_b || ag->rows_per_rank <= 0 || ag->rows_per_rank % kBM ||
        ag->rows_per_rank * ag->world != a->M)
      return kErrBadShape;
    a_ptr = ag->a_peer[ag->rank];
  }
  p.M = a->M; p.N = a->N; p.K = a->K;
  p.C = a->C; p.ldc = a->ldc;
  p.bias = a->bias; p.bias_f32 = a->bias_f32;
  p.residual = static_cast<const __nv_bfloat16*>(a->residual); p.ldr = a->ldr;
  p.aux_out = static_cast<__nv_bfloat16*>(a->aux_out); p.ld_aux_out = a->ld_aux_out;
  p.aux_in = static_cast<const __nv_bfloat16*>(a->aux_in); p.ld_aux_in = a->ld_aux_in;
  p.act = a->act; p.out_f32 = a->out_f32; p.accumulate = a->accumulate; p.alpha = a->alpha;
  if (p.act >= 11 && !p.aux_in) return kErrBadShape;
  if (p.act == 5 && !p.aux_out) p.act = 2;

  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool tc_ok = !a->force_simt && !a->a_f32 && !a->b_f32 && a->K > 0 && al16(a_ptr) && al16(a->B) &&
                     (a->lda % 8 == 0) && (a->ldb % 8 == 0);
  p.vec_ok = al16(p.C) && (p.ldc % 8 == 0) && (!p.bias || al16(p.bias)) &&
             (!p.residual || (al16(p.residual) && p.ldr % 8 == 0)) &&
             (!p.aux_out || (al16(p.aux_out) && p.ld_aux_out % 8 == 0)) &&
             (!p.aux_in || (al16(p.aux_in) && p.ld_aux_in % 8 == 0));

  if (ar) {
    // The all-reduce epilogue exists on the tensor-core path only and moves whole 16-byte groups.
    if (!tc_ok || !p.vec_ok || (a->N % 8) || a->out_f32 || a->act || a->aux_out || a->aux_in || a->accumulate)
      return kErrUnsupported;
    if (ar->world < 1 || ar->world > kMaxRanks || ar->rank < 0 || ar->rank >= ar->world) return kErrBadShape;
    if (ar->mode == 1 && (a->M % (ar->world * kBM))) return kErrBadShape;   // whole row tiles per shard
  }
  if (ag && (!tc_ok || a->splits > 1)) return kErrUnsupported;
  if (!tc_ok) {
    p.tiles_m = p.tiles_n = p.num_kb = 0;
    p.splits = 1; p.kb_per_split = 0; p.ws = nullptr; p.counters = nullptr;
    dim3 grid((unsigned)((a->N + 63) / 64), (unsigned)((a->M + 63) / 64));
    const long long sam = a->trans_a ? 1 : a->lda, sak = a->trans_a ? a->lda : 1;
    const long long sbk = a->trans_b ? 1 : a->ldb, sbn = a->trans_b ? a->ldb : 1;
    if (a->a_f32 && a->b_f32)
      gemm_simt_kernel<float, float><<<grid, 256, 0, stream>>>((const float*)a->A, sam, sak, (const float*)a->B, sbk, sbn, p);
    else if (!a->a_f32 && !a->b_f32)
      gemm_simt_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)a->A, sam, sak, (const __nv_bfloat16*)a->B, sbk, sbn, p);
    else if (a->a_f32)
      gemm_simt_kernel<float, __nv_bfloat16><<<grid, 256, 0, stream>>>((const float*)a->A, sam, sak, (const __nv_bfloat16*)a->B, sbk, sbn, p);
    else
      gemm_simt_kernel<__nv_bfloat16, float><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)a->A, sam, sak, (const float*)a->B, sbk, sbn, p);
    return counted(1, (int)cudaGetLastError());
  }

  // Tile width and split-K factor from a small cost model (unit: the time of one 128x256x64 k-block).
  //   a CTA runs ceil(units / SMs) units back to back; a unit costs its k-blocks (a 128-wide tile moves as many bytes
  //   for half the math, so its k-block counts 0.75) plus a fixed prologue/epilogue, plus the partial-tile round
  //   trip when K is split.
  const int num_kb = (a->K + kBK - 1) / kBK;
  const int tm = (a->M + kBM - 1) / kBM;
  // CTA pairs (256-row tiles shared by two SMs) for every plain GEMM with at least two row tiles; the fused
  // tensor-parallel variants keep single CTAs.  DPTB_GEMM_PAIR=0 switches pairs off (for comparisons).
  static const bool pairs_enabled = [] {
    const char* e = getenv("DPTB_GEMM_PAIR");
    return !(e && e[0] == '0');
  }();
  // A pair's epilogue leaves through tile stores: bf16 output, every per-element buffer describable by a tensor map
  // (16-byte aligned, strides multiples of 16 bytes), at most one per-element input, and a pre-activation copy not
  // combined with an input (a warp's two staging blocks cover either case).
  const int epi_inputs = (p.act >= 11 ? 1 : 0) + (p.residual ? 1 : 0) + (p.accumulate ? 1 : 0);
  const bool tile_store_ok = !p.out_f32 && p.vec_ok && !(p.bias && p.bias_f32) && (a->N % 8) == 0 && epi_inputs <= 1 &&
                             !(epi_inputs == 1 && p.aux_out);
  const bool pair = pairs_enabled && !ar && !ag && tm >= 2 && tile_store_ok;
  // Work units run on `sms` CTAs, or on sms / 2 pairs, each pair taking two row tiles at a time.
  const int sms = pair ? sm_count() / 2 : sm_count();
  const int tm_sched = pair ? (tm + 1) / 2 : tm;
  int bn = a->bn, splits = a->splits;
  {
    double best = 1e30;
    int best_bn = 128, best_sp = 1;
    for (int cand_bn = 128; cand_bn <= 256; cand_bn += 128) {
      if (a->bn == 128 || a->bn == 256) { if (cand_bn != a->bn) continue; }
      if (cand_bn == 256 && a->N <= 128) continue;
      const int tiles = tm * ((a->N + cand_bn - 1) / cand_bn);
      const int sched_tiles = tm_sched * ((a->N + cand_bn - 1) / cand_bn);
      for (int sp = 1; sp <= 8; ++sp) {
        if (a->splits >= 1 && sp != a->splits) continue;
        if ((ar || ag) && sp > 1) break;
        if (sp > 1) {
          if (!a->ws || !a->counters || tiles > a->num_counters) break;
          if ((long long)tiles * sp * cand_bn * kBM * 4 > a->ws_bytes) break;
          if (num_kb / sp < 4) break;
        }
        const int kbs = (num_kb + sp - 1) / sp;
        const long long units = (long long)sched_tiles * sp;
        const double waves = (double)((units + sms - 1) / sms);
        const double per_kb = cand_bn == 256 ? 1.0 : 0.75;
        // (the fold of a 256-wide tile is serial in its last CTA: measured on 768 x 768 x 16384, 8 splits of 256-wide tiles
        // took 48 us against 42 us for 4 splits of 128-wide ones)
        const double fixed = (cand_bn == 256 ? 8.0 : 5.0) + (sp > 1 ? (cand_bn == 256 ? 8.0 + 2.5 * sp : 4.0 + 1.0 * sp) : 0.0);
        const double cost = waves * (kbs * per_kb + fixed);
        if (cost < best) { best = cost; best_bn = cand_bn; best_sp = sp; }
      }
    }
    bn = best_bn;
    splits = best_sp;
  }
  p.tiles_m = tm;
  p.tiles_n = (a->N + bn - 1) / bn;
  p.num_kb = num_kb;
  p.splits = splits;
  p.kb_per_split = (num_kb + splits - 1) / splits;
  if ((long long)(splits - 1) * p.kb_per_split >= num_kb) {  // keep every split non-empty
    splits = (num_kb + p.kb_per_split - 1) / p.kb_per_split;
    p.splits = splits;
  }
  p.ws = static_cast<float*>(a->ws);
  p.counters = a->counters;
  if (ar) {
    const long long tiles = (long long)p.tiles_m * p.tiles_n;
    if (p.splits != 1 || tiles > ar->max_tiles || tiles * bn * kBM > ar->partial_elems) return kErrTooLarge;
    p.ar.world = ar->world; p.ar.rank = ar->rank;
    p.ar.use_nvls = (ar->use_nvls && ar->mc_partial && ar->mc_out) ? 1 : 0;
    p.ar.partial = static_cast<__nv_bfloat16*>(ar->partial);
    p.ar.mc_partial = static_cast<const __nv_bfloat16*>(ar->mc_partial);
    p.ar.mc_out = static_cast<__nv_bfloat16*>(ar->mc_out);
    for (int r = 0; r < kMaxRanks; ++r) {
      p.ar.peer_partial[r] = static_cast<const __nv_bfloat16*>(ar->peer_partial[r]);
      p.ar.out_peer[r] = static_cast<__nv_bfloat16*>(ar->out_peer[r]);
      p.ar.flags_peer[r] = static_cast<uint32_t*>(ar->flags_peer[r]);
    }
    p.ar.max_tiles = ar->max_tiles;
    p.ar.epoch = static_cast<uint32_t*>(ar->epoch);
    p.ar.exit_counter = static_cast<unsigned int*>(ar->exit_counter);
    p.ar.mode = ar->mode == 1 ? 1 : 0;
    p.ar.rows_per_rank = a->M / ar->world;
  }
  if (ag) {
    p.ag.world = ag->world;
    p.ag.rank = ag->rank;
    p.ag.tiles_per_rank = (int)(ag->rows_per_rank / kBM);
    p.ag.ready = static_cast<const uint32_t*>(ag->ready);
    p.ag.epoch = static_cast<const uint32_t*>(ag->epoch);
    p.row_epi = (!p.out_f32 && p.vec_ok && !(p.bias && p.bias_f32)) ? 1 : 0;
    TmapSet peers;
    for (int r = 0; r < kMaxRanks; ++r) {
      const int src = r < ag->world ? r : ag->rank;
      if (!al16(ag->a_peer[src])) return kErrBadShape;
      const int rc_a = encode_tmap_2d_bf16(&peers.m[r], ag->a_peer[src], (uint64_t)a->K, (uint64_t)ag->rows_per_rank,
                                           (uint64_t)a->lda * 2, 64, kBM);
      if (rc_a) return rc_a;
    }
    CUtensorMap tmBg;
    const int rc_b = encode_tmap_2d_bf16(&tmBg, a->B, (uint64_t)a->K, (uint64_t)a->N, (uint64_t)a->ldb * 2, 64, (uint32_t)bn);
    if (rc_b) return rc_b;
    return &gemm_launch_ag ? gemm_launch_ag(bn, peers, tmBg, p, stream) : kErrUnsupported;
  }

  CUtensorMap tmA, tmB;
  int rc;
  if (a->trans_a) rc = encode_tmap_2d_bf16(&tmA, a->A, (uint64_t)a->M, (uint64_t)a->K, (uint64_t)a->lda * 2, 64, 64);
  else            rc = encode_tmap_2d_bf16(&tmA, a->A, (uint64_t)a->K, (uint64_t)a->M, (uint64_t)a->lda * 2, 64, kBM);
  if (rc) return rc;
  if (a->trans_b) rc = encode_tmap_2d_bf16(&tmB, a->B, (uint64_t)a->K, (uint64_t)a->N, (uint64_t)a->ldb * 2, 64,
                                           (uint32_t)(pair ? bn / 2 : bn));
  else            rc = encode_tmap_2d_bf16(&tmB, a->B, (uint64_t)a->N, (uint64_t)a->K, (uint64_t)a->ldb * 2, 64, 64);
  if (rc) return rc;

  // bf16 outputs take the row-per-thread register epilogue (DPTB_GEMM_STAGED_EPILOGUE=1 keeps the staged one, for
  // comparisons); 32-byte accesses when every per-element buffer allows them.
  static const bool staged_only = [] {
    const char* e = getenv("DPTB_GEMM_STAGED_EPILOGUE");
    return e && e[0] == '1';
  }();
  p.row_epi = (!ar && !staged_only && !p.out_f32 && p.vec_ok && !(p.bias && p.bias_f32)) ? 1 : 0;
  if (p.row_epi) {
    auto wide_ok = [](const void* q, long long ld) { return (reinterpret_cast<uintptr_t>(q) & 31) == 0 && ld % 16 == 0; };
    if (wide_ok(p.C, p.ldc) && (!p.residual || wide_ok(p.residual, p.ldr)) &&
        (!p.aux_out || wide_ok(p.aux_out, p.ld_aux_out)) && (!p.aux_in || wide_ok(p.aux_in, p.ld_aux_in)))
      p.row_epi = 2;
  }

  // CTA pairs with a bf16 output take the tile-store epilogue when every per-element buffer can be described by a
  // tensor map (16-byte aligned, row strides multiples of 16 bytes: vec_ok), at most one per-element input is read
  // and a pre-activation copy is not combined with an input (the two staging blocks of a warp cover either case).
  EpiMaps em;
  if (pair && p.splits == 1) {
    const int inputs = epi_inputs;
    {
      const void* in_ptr = p.act >= 11 ? (const void*)p.aux_in : (p.residual ? (const void*)p.residual : p.C);
      const long long in_ld = p.act >= 11 ? p.ld_aux_in : (p.residual ? p.ldr : p.ldc);
      int e = encode_tmap_2d_bf16(&em.c, p.C, (uint64_t)a->N, (uint64_t)a->M, (uint64_t)p.ldc * 2, 64, 32);
      if (!e) e = p.aux_out ? encode_tmap_2d_bf16(&em.aux, p.aux_out, (uint64_t)a->N, (uint64_t)a->M,
                                                  (uint64_t)p.ld_aux_out * 2, 64, 32)
                            : (em.aux = em.c, 0);
      if (!e) e = inputs ? encode_tmap_2d_bf16(&em.in, in_ptr, (uint64_t)a->N, (uint64_t)a->M, (uint64_t)in_ld * 2, 64, 32)
                         : (em.in = em.c, 0);
      if (e) return e;
      p.row_epi = 3;
    }
  }
  if (p.row_epi != 3) em.c = em.aux = em.in = tmA;   // unused by the kernel, but kernel parameters must be initialised

  const bool amn = a->trans_a != 0, bmn = a->trans_b == 0;
  const auto launch = amn ? (bmn ? &gemm_launch_tt : &gemm_launch_tn) : (bmn ? &gemm_launch_nn : &gemm_launch_nt);
  return launch ? launch(pair, bn, tmA, tmB, em, p, stream) : kErrUnsupported;
}

extern "C" int dptb_gemm(const DptbGemmArgs* a, void* stream_v) { return gemm_impl(a, nullptr, nullptr, stream_v); }
// Row-parallel Linear of a tensor-parallel group in ONE kernel: tcgen05 GEMM of this rank's K-slice, then the sum over
// ranks (+ bias, + residual) through NVLink peer memory, delivered to every rank's `out`.  Every rank must call it with
// the same shapes; C of the argument block is ignored (the result goes to ar->out_peer / ar->mc_out with row stride ldc).
extern "C" int dptb_gemm_allreduce(const DptbGemmArgs* a, const DptbTpArArgs* ar, void* stream_v) {
  if (!ar) return kErrBadShape;
  return gemm_impl(a, ar, nullptr, stream_v);
}
// Column-parallel Linear on a row-sharded input in ONE kernel: row tile i of A is read by TMA straight from the
// symmetric buffer of the rank that owns those rows, once that rank's dptb_tp_signal has published the shard; the
// output [M, N] (this rank's slice of the features, all rows) is local.  A of the argument block is ignored.
extern "C" int dptb_allgather_gemm(const DptbGemmArgs* a, const DptbTpAgArgs* ag, void* stream_v) {
  if (!ag) return kErrBadShape;
  return gemm_impl(a, nullptr, ag, stream_v);
}

// Publishes "this rank's shard is complete" to every peer: flag word [rank] of each peer's `ready` array and the local
// launch counter both become *epoch + 1.  Runs after the kernel that wrote the shard, in stream order.
struct DptbTpSignalArgs {
  int world, rank;
  void* ready_peer[kMaxRanks];   // every rank's flag array [kMaxRanks]
  void* epoch;                   // local launch counter
};
namespace dptb {
struct SignalParams {
  int world, rank;
  uint32_t* ready_peer[kMaxRanks];
  uint32_t* epoch;
};
__global__ void tp_shard_signal_kernel(const SignalParams s) {
  const uint32_t e = *reinterpret_cast<volatile uint32_t*>(s.epoch) + 1u;
  __threadfence_system();   // the shard written by earlier kernels of this stream is visible system-wide first
  if ((int)threadIdx.x < s.world) st_release_sys(s.ready_peer[threadIdx.x] + s.rank, e);
  __syncwarp();
  if (threadIdx.x == 0) *s.epoch = e;
}
}  // namespace dptb
extern "C" int dptb_tp_signal(const DptbTpSignalArgs* a, void* stream_v) {
  if (!a || a->world < 1 || a->world > kMaxRanks) return kErrBadShape;
  SignalParams s;
  s.world = a->world;
  s.rank = a->rank;
  for (int r = 0; r < kMaxRanks; ++r) s.ready_peer[r] = static_cast<uint32_t*>(a->ready_peer[r]);
  s.epoch = static_cast<uint32_t*>(a->epoch);
  tp_shard_signal_kernel<<<1, 32, 0, static_cast<cudaStream_t>(stream_v)>>>(s);
  return counted(1, (int)cudaGetLastError());
}

// Stream-ordered wait for the peers' shards: returns once every other rank's "shard ready" flag in THIS rank's flag
// array has reached this rank's own publication count (so it runs after this rank's dptb_tp_signal).  Each wait is
// bounded; one that runs out is recorded in the status word and the kernel returns all the same.  What follows it on
// the stream (copies of the peers' shards into local memory) then sees complete shards.
namespace dptb {
__global__ void tp_wait_ready_kernel(const uint32_t* ready, const uint32_t* epoch, int world, int rank) {
  const uint32_t e = *reinterpret_cast<const volatile uint32_t*>(epoch);
  const int src = threadIdx.x;
  if (src < world && src != rank) wait_flag_ge(ready + src, e);
}
}  // namespace dptb
// One device-to-device copy on the stream by the copy engines (no SM is taken from the GEMM that runs beside it);
// either pointer may be peer-mapped memory.
extern "C" int dptb_copy_async(void* dst, const void* src, long long nbytes, void* stream_v) {
  if (nbytes <= 0) return 0;
  if (!dst || !src) return kErrBadShape;
  return (int)cudaMemcpyAsync(dst, src, (size_t)nbytes, cudaMemcpyDeviceToDevice, static_cast<cudaStream_t>(stream_v));
}
extern "C" int dptb_tp_wait_ready(const void* ready, const void* epoch, int world, int rank, void* stream_v) {
  if (!ready || !epoch || world < 1 || world > kMaxRanks || rank < 0 || rank >= world) return kErrBadShape;
  tp_wait_ready_kernel<<<1, 32, 0, static_cast<cudaStream_t>(stream_v)>>>(
      static_cast<const uint32_t*>(ready), static_cast<const uint32_t*>(epoch), world, rank);
  return counted(1, (int)cudaGetLastError());
}

// Status word access ------------------------------------------------------------------------------
// Folds the blocks of all translation units: the first non-zero code (with its detail) and the total number of
// waits that ran out.
extern "C" int dptb_status_read(int* out4) {
  out4[0] = out4[1] = out4[2] = out4[3] = 0;
  for (int i = 0; i < g_num_status_blocks; ++i) {
    int b[4] = {0, 0, 0, 0};
    const int rc = g_status_blocks[i](b, 0);
    if (rc) return rc;
    if (out4[0] == 0 && b[0] != 0) { out4[0] = b[0]; out4[1] = b[1]; }
    out4[2] += b[2];
  }
  return 0;
}
extern "C" int dptb_status_clear() {
  for (int i = 0; i < g_num_status_blocks; ++i) {
    const int rc = g_status_blocks[i](nullptr, 1);
    if (rc) return rc;
  }
  return 0;
}

extern "C" long long dptb_launch_count() { return launch_counter(); }
extern "C" void dptb_launch_count_reset() { launch_counter() = 0; }
