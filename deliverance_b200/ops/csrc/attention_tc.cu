// Paged flash attention for prefill on the 5th-generation tensor cores (tcgen05 / TMEM / TMA).
//
// One CTA per (256 query rows of one sequence, query head): two 128-row query tiles that share every K / V tile (one tile when fewer
// than 129 rows are left, or for head_dim 256, whose accumulator leaves no room for a second one). Keys go by in tiles of 64.
//   warp 1            = TMA producer: the Q tiles once (D / 64 boxes of 128 rows x 64 columns each), then per key tile the K and V rows
//                       of its cache pages (a page slice of one KV head is `page` rows x D contiguous bf16 = D / 64 boxes of up to 64
//                       rows x 64 columns), all into 128-byte-swizzled shared memory, completion on mbarriers, 4 stages (2 for D = 256);
//                       the copies of a tile are spread over the warp's lanes;
//   warp 0, one lane  = issues S = Q K^T for every (key tile, query tile): both operands from shared memory, K-major, the
//                       accumulator is one of the query tile's two 64-column score slots in tensor memory;
//   warp 2, one lane  = issues O += P V: P from tensor memory as the A operand, V from shared memory as an MN-major B operand;
//   warps 4-7 (8-11)  = softmax of query tile 0 (1): thread r owns query row r (TMEM lane r): tcgen05.ld of the 64 scores, mask
//                       (causal / sliding window / context end), optional logit soft-cap, running maximum and sum in registers, rescale
//                       of the O accumulator in tensor memory when the maximum has moved by more than 2^8, P written back over the
//                       scores as packed bf16 (tcgen05.st), finally O / l to global memory.
// Tensor memory (512 columns): score slots at [0, 256) = (query tile, slot) x 64, accumulators at 256 + query tile x D.
// Why two issuing threads: a tcgen05.mma holds its thread until the pipe accepts it and the pipe queues almost nothing, so the tensor
// cores idle whenever their issuer waits on a barrier (even a complete one costs a few hundred cycles) or walks its loop; with the
// Q K^T and the P V streams on threads of their own, one feeds the pipe while the other waits. Measured on the way here (B200, 32 query
// / 8 KV heads of 128, 2 x 8192 tokens causal): one issuing warp whose 32 lanes all wait and vote 442 TFLOP/s, the same loop on one
// lane 443, two issuing threads 729; a single thread issuing all copies of a tile 265, the lanes of the warp 733.
// Every wait is bounded (common.cuh); on expiry the CTA records a status word, skips its stores, lets its copies and MMAs drain
// (bounded), frees tensor memory and returns; CTAs that start after a recorded failure leave at once.
//
// Three layouts share the kernel (template parameters LATENT, KM):
//   paged   q [T, H * dk], K and V rows in the paged cache, GQA groups; the real widths dk and dv may be smaller than DK and DV (multiples
//           of 8): tensor-map bounds fill the columns behind a cache row with zeros, and query columns that reach into the next head meet
//           zeros. The first `keep_first` keys stay visible beside a sliding window (their key tiles are listed in front of the window's),
//           `sink` adds a score per head without a value to the softmax, the epilogue may multiply with a sigmoid output gate per column or
//           per head and a constant;
//   latent  keys and values expanded from the latent cache into flat rows (latent.cu): per head kn columns of an unrotated key part, one
//           rotated key part shared by all heads (its own tensor map: it is copied behind the head's columns of every K tile, never
//           materialised per head), DV columns of value. Key 0 of a sequence is its row kv_row0 of those buffers. The epilogue multiplies
//           with a sigmoid output gate and stores the dv real columns of every head.
// Both take DK (query / key columns) and DV (value columns) as multiples of 64.
//
//   wide    (KM > 0) attention with mixed scores, the mixing moved to the query side (ops/grouped.py): a row holds the heads of all KV heads side by side,
//           a query head's keys are the WHOLE row, its values the dv columns of its own KV head. The visible cache rows have been gathered into flat
//           buffers (key 0 of a sequence is row kv_row0), key rows padded with zeros to 64-column blocks, so that one copy fetches 64 keys x several
//           blocks: with a copy per cache page and block the copy engine sets the pace (20 copies per tile of 512 columns: 3.4 us). KM = 3: whole key
//           tiles, rows of up to 256 columns. Wider rows go by in pieces of 128 columns: KM = 1, the query tile of up to 512 columns stays in shared
//           memory; KM = 2, the query's pieces travel with the keys' pieces, from L2. With KM = 1, 2 and QT = 2 there is ONE query tile, and the two
//           softmax groups take its key tiles in turn, each with an accumulator, maximum and sum of its own; they meet in the epilogue. Warps 0 and 3
//           then issue the Q K^T of one group's tiles each, from halves of the key ring: a group of eight MMAs behind a wait costs its thread about a
//           thousand cycles, twice the MMAs themselves (one thread 337 us for 16 heads over rows of 512 columns, whatever the depth of the ring).
//
// Replaces the reference's packed prefill attention (core/.../generator/CausalSelfAttention.java:458-502: per head QK^T GEMM over
// the visible pages, causal scaled softmax with optional soft-cap, saxpy with V).
#include <stdexcept>
#include <string>

#include "common.cuh"
#include "gemm_api.h"

namespace dlv {

void encode_map_kchunks(CUtensorMap* map, const void* base, uint64_t rows, uint64_t K, uint64_t pitch_bytes, uint32_t box_rows, uint32_t chunks = 2);
void encode_map_2d(CUtensorMap* map, int dtype_code, const void* base, uint64_t rows, uint64_t cols, uint64_t pitch_bytes, uint32_t box_rows,
                   uint32_t box_cols, int swizzle_code);

struct AttnTcParams {
  const int* block_tables;
  int bt_stride;
  const int* q_start;
  const int* q_len;
  const int* ctx_lens;
  const int* tile_seq;
  const int* tile_q0;
  __nv_bfloat16* out;  // [T, H * D]
  int H, KV, page_size;
  float scale, softcap;
  int window, causal;
  int keep_first;
  const float* sink;           // [H] (nullptr: none)
  int dk;                      // query columns per head in q (paged layout: also the width of a K row)
  int* status;
  int dv;                      // real value columns per head
  long long out_pitch;         // row pitch of out
  const int* kv_row0;          // latent layout: [sequences] row of key 0 in the expanded buffers
  int kn_blocks;               // latent layout: 64-column blocks of the per-head key part (the blocks behind it come from the shared part)
  const __nv_bfloat16* gate;   // gate logits [T, gate_pitch], head h at column h * dv, or one per head at column h (nullptr: no gate)
  long long gate_pitch;
  int gate_heads;
  float out_mult;
  int k_subs;                  // wide layout: 64-column blocks of a key row
};

// MN-major shared-memory descriptor (128-byte swizzle): the operand tile is stored as rows of the K dimension, each row 64 elements of
// the MN dimension (128 bytes); 8 rows form a 1 KB swizzle atom. lbo: bytes between atoms along MN (the next 64 columns), sbo: bytes
// between atoms along K (the next 8 rows).
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>((lbo_bytes >> 4) & 0x3FFFu) << 16;
  d |= static_cast<uint64_t>((sbo_bytes >> 4) & 0x3FFFu) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
// kind::f16, bf16 x bf16 -> fp32, A K-major, B MN-major
__host__ __device__ constexpr uint32_t umma_idesc_bf16_bmn(int m, int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (0u << 15) | (1u << 16) | (static_cast<uint32_t>(n >> 3) << 17) | (static_cast<uint32_t>(m >> 4) << 24);
}
__device__ __forceinline__ void tmem_ld_x32(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
        "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
}
__device__ __forceinline__ void tmem_st_x32(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
      "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]),
      "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

constexpr int kAtBM = 128, kAtBN = 64;  // query rows per score tile / keys per tile
constexpr int kAtPiece = 2, kAtResident = 8;  // KM = 1, 2: 64-column blocks per piece of a key row; most blocks of a query tile that stays in shared memory

// KM = 1, 2 (one query tile): a K stage is one piece of a key tile, with KM = 2 behind the query's piece
template <int DV, int QT, int KM>
struct AttnTcWideSmem {
  static constexpr int kTileQ = kAtBM * 128 * kAtPiece;  // bytes of a query piece
  static constexpr int kTileK = kAtBN * 128 * kAtPiece + (KM == 2 ? kTileQ : 0);
  static constexpr int kOffKeys = KM == 2 ? kTileQ : 0;  // the keys inside a stage
  static constexpr int kTileV = kAtBN * 128 * (DV / 64);
  static constexpr int kStagesV = 2;
  static constexpr int kOffK = KM == 1 ? kAtResident * kAtBM * 128 : 0;
  static constexpr int kRoom = 227 * 1024 - 512 - 1024 - kOffK - kStagesV * kTileV;
  static constexpr int kFit = kRoom / kTileK;
  static constexpr int kStages = kFit >= 4 ? 4 : kFit;
  static constexpr int kOffV = kOffK + kStages * kTileK;
  static constexpr int kOffCtrl = kOffV + kStagesV * kTileV;
  static constexpr int kBytes = kOffCtrl + 512 + 1024;
  static constexpr int kThreads = 128 + 128 * QT;
  static constexpr int kSubK = 0, kSubV = DV / 64;
  static_assert(kStages >= 2 && (QT == 1 || kStages == 4) && DV % 64 == 0 && kBytes > 118 * 1024 && kBytes <= 227 * 1024 && 256 + QT * DV <= 512, "attention tile does not fit");
};

template <int DK, int DV, int QT>
struct AttnTcSmem {
  static constexpr int kSubK = DK / 64, kSubV = DV / 64;  // 64-column sub-tiles per operand tile
  static constexpr int kTileQ = kAtBM * 128 * kSubK;      // bytes of a [128 rows][DK] bf16 query tile
  static constexpr int kTileK = kAtBN * 128 * kSubK;      // bytes of a [64 keys][DK] bf16 K tile
  static constexpr int kTileV = kAtBN * 128 * kSubV;
  static constexpr int kRoom = 227 * 1024 - 512 - 1024 - QT * kTileQ;  // barriers + alignment slack
  static constexpr int kFit = kRoom / (kTileK + kTileV);
  static constexpr int kStages = kFit >= 4 ? 4 : kFit, kStagesV = kStages, kOffKeys = 0;
  static constexpr int kOffK = QT * kTileQ;
  static constexpr int kOffV = kOffK + kStages * kTileK;
  static constexpr int kOffCtrl = kOffV + kStages * kTileV;
  static constexpr int kNeed = kOffCtrl + 512 + 1024;
  // every CTA allocates all 512 tensor-memory columns, so two CTAs must never share an SM: ask for more than half of its shared memory
  static constexpr int kBytes = kNeed > 118 * 1024 ? kNeed : 118 * 1024;
  static constexpr int kThreads = 128 + 128 * QT;  // warp 0 issues Q K^T, warp 1 the copies, warp 2 issues P V, warp 3 idles, warps 4.. softmax
  static_assert(kStages >= 2 && DK % 64 == 0 && DV % 64 == 0, "attention tile does not fit");
  static_assert(256 + QT * DV <= 512, "score slots and accumulators exceed tensor memory");
};

// eight columns times the sigmoid of their gate logits
__device__ __forceinline__ void gate8(float* w, const uint4& gv) {
  const uint32_t* gu = reinterpret_cast<const uint32_t*>(&gv);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 g2 = unpack_bf162(gu[e]);
    w[2 * e] /= 1.f + __expf(-g2.x);
    w[2 * e + 1] /= 1.f + __expf(-g2.y);
  }
}

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float y;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(y) : "f"(a), "f"(b), "f"(c));
  return y;
}

// f <- cap * tanh(f * a) for a thread's row of scores. Where all of a warp's arguments are small (scores far below the cap, the usual case)
// the series of the hyperbolic tangent around 0 up to x^11 is exact to fp32 rounding and needs no special-function unit, which is what
// limits the loop around it; otherwise tanh(x) = 1 - 2 / (e^(2 x) + 1), with an absolute error of a few units in the last place of 1.
__device__ __forceinline__ void softcap_tile(float (&f)[kAtBN], float a, float cap) {
  float mx = 0.f;
#pragma unroll
  for (int i = 0; i < kAtBN; ++i) mx = fmaxf(mx, fabsf(f[i]));
  if (__all_sync(0xffffffffu, mx * a < 0.35f)) {
    const float ac = a * cap, a2 = a * a;
#pragma unroll
    for (int i = 0; i < kAtBN; ++i) {
      const float x2 = f[i] * f[i] * a2;
      float s = fmaf(x2, -1382.f / 155925.f, 62.f / 2835.f);
      s = fmaf(x2, s, -17.f / 315.f);
      s = fmaf(x2, s, 2.f / 15.f);
      s = fmaf(x2, s, -1.f / 3.f);
      s = fmaf(x2, s, 1.f);
      f[i] = f[i] * ac * s;
    }
  } else {
    const float k = 2.f * 1.4426950408889634f * a;
#pragma unroll
    for (int i = 0; i < kAtBN; ++i) f[i] = cap - __fdividef(2.f * cap, ex2_approx(f[i] * k) + 1.f);
  }
}

template <int DK, int DV, int QT, int KM>
struct AttnTcLayout {
  using T = AttnTcSmem<DK, DV, QT>;
};
template <int DV, int QT, int KM>
struct AttnTcLayout<0, DV, QT, KM> {
  using T = AttnTcWideSmem<DV, QT, KM>;
};

template <int DK, int DV, int QT, bool LATENT, int KM = 0>
__global__ void __launch_bounds__(AttnTcLayout<DK, DV, QT, KM>::T::kThreads, 1)
    prefill_attn_tc_kernel(const __grid_constant__ CUtensorMap map_q,  // [T, H * DK], box 128 x 64
                           const __grid_constant__ CUtensorMap map_k,  // paged [pages * KV * page, DK], box min(page, 64) x 64; latent [rows, H * kn]
                           const __grid_constant__ CUtensorMap map_v,  // paged as K; latent [rows, H * DV], box 64 x 64
                           const __grid_constant__ CUtensorMap map_r,  // latent: shared key part [rows, DK - kn], box 64 x 64 (paged: unused)
                           const AttnTcParams p) {
  using L = typename AttnTcLayout<DK, DV, QT, KM>::T;
  constexpr int NS = L::kStages, NSV = L::kStagesV, SUBK = L::kSubK, SUBV = L::kSubV;
  constexpr bool PIECES = KM == 1 || KM == 2;
  const int pieces = PIECES ? (p.k_subs + kAtPiece - 1) / kAtPiece : 1;  // K stages per key tile
  constexpr int kProducer = 1, kIssuer = 0, kIssuerPV = 2, kIssuer2 = 3;  // (kIssuer2: SPLIT, the second softmax group's Q K^T)
  extern __shared__ uint8_t at_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(at_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bar_q = reinterpret_cast<uint64_t*>(smem + L::kOffCtrl);
  uint64_t* bar_k_full = bar_q + 1;        // [4] K tile landed
  uint64_t* bar_v_full = bar_k_full + 4;   // [4] V tile landed
  uint64_t* bar_k_empty = bar_v_full + 4;  // [4] every Q K^T of the tile has retired
  uint64_t* bar_v_empty = bar_k_empty + 4; // [4] every P V of the tile has retired
  uint64_t* bar_s_full = bar_v_empty + 4;  // [2 query tiles][2 slots] scores complete
  uint64_t* bar_p_full = bar_s_full + 4;   // [2][2] probabilities written over the scores
  uint64_t* bar_pv_done = bar_p_full + 4;  // [2][2] the P V that read the slot's probabilities has retired
  uint64_t* bar_o_final = bar_pv_done + 4;
  uint64_t* bar_drain = bar_o_final + 1;    // [3] an issuing thread's MMAs have retired (only used when a wait ran out)
  uint64_t* bar_ml = bar_drain + 3;         // SPLIT: maxima and sums of both softmax groups are in shared memory
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar_ml + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // a CTA that starts after another one of this or an earlier launch has recorded a failed wait leaves at once: one stuck tile
  // must not make every later tile sit out its own time limit
  if (__syncthreads_or(threadIdx.x == 0 && *reinterpret_cast<volatile int*>(p.status) != 0)) return;
  // heavy tiles first: inside a sequence the late query tiles see the most keys, and the host lists tiles in ascending order
  const int tile = static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x);
  const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile], h = blockIdx.y;
  const int kvh = h / (p.H / p.KV);
  const int qs = p.q_start[seq], ql = p.q_len[seq], ctx = p.ctx_lens[seq];
  const int pos0 = ctx - ql;  // position of the sequence's first query row
  constexpr bool SPLIT = PIECES && QT == 2;  // one query tile, its key tiles alternate between the softmax groups
  const int rows_all = min((SPLIT ? 1 : QT) * kAtBM, ql - q0);
  const bool two = QT == 2 && (SPLIT || rows_all > kAtBM);  // two query tiles share every K / V tile
  // key tiles [a, b) each query tile sees
  int rows_q[2], first_q[2], a_q[2], b_q[2];
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const int behind = SPLIT ? 0 : q * kAtBM;
    rows_q[q] = max(0, min(kAtBM, rows_all - behind));
    first_q[q] = pos0 + q0 + behind;
    const int last_pos = p.causal ? first_q[q] + rows_q[q] - 1 : ctx - 1;
    const int key_hi = min(ctx, last_pos + 1);
    const int key_lo = p.window > 0 ? max(0, first_q[q] - p.window + 1) : 0;
    a_q[q] = key_lo / kAtBN;
    b_q[q] = rows_q[q] > 0 ? (key_hi + kAtBN - 1) / kAtBN : a_q[q];
  }
  const int a0 = a_q[0], b0 = b_q[0], a1 = a_q[1], b1 = two ? b_q[1] : a_q[1];
  // key tiles this CTA loads, in this order: those that hold kept first tokens in front of the window, then [lo, hi)
  const int kept_tiles = (min(p.keep_first, ctx) + kAtBN - 1) / kAtBN;
  const int lo = a0, hi = two ? max(b0, b1) : b0;
  const int n_kept = min(kept_tiles, lo);
  const int n_tiles = n_kept + hi - lo;
  auto tile_at = [&](int u) { return u < n_kept ? u : lo + u - n_kept; };

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(bar_q), 1);
    for (int s = 0; s < 4; ++s) {
      mbar_init(smem_u32(&bar_k_full[s]), 1);
      mbar_init(smem_u32(&bar_v_full[s]), 1);
      mbar_init(smem_u32(&bar_k_empty[s]), 1);
      mbar_init(smem_u32(&bar_v_empty[s]), 1);
      mbar_init(smem_u32(&bar_s_full[s]), 1);
      mbar_init(smem_u32(&bar_p_full[s]), 4);
      mbar_init(smem_u32(&bar_pv_done[s]), 1);
    }
    mbar_init(smem_u32(&bar_drain[0]), 1);
    mbar_init(smem_u32(&bar_drain[1]), 1);
    mbar_init(smem_u32(&bar_drain[2]), 1);
    mbar_init(smem_u32(bar_o_final), 1);
    mbar_init(smem_u32(bar_ml), 8);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
    if (LATENT) tma_prefetch_desc(&map_r);
  }
  constexpr uint32_t kTmemCols = 512;
  if (warp == kIssuer) tmem_alloc(smem_u32(tmem_slot), kTmemCols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  constexpr uint32_t kColS = 0, kColO = 256;  // score slot b of query tile q at kColS + (2 q + b) 64, accumulator of query tile q at kColO + q DV
  pdl_wait();
  pdl_trigger();

  if (warp == kProducer) {
    // ---------------- TMA producer ----------------
    // One thread can start a tensor copy only every few hundred nanoseconds, whatever its size, and a key tile is several copies
    // (pages x D / 64 column blocks, for K and for V): the copies of a tile are spread over the lanes of the warp.
    if (KM == 1) {
      if (lane == 0) mbar_expect_tx(smem_u32(bar_q), pieces * L::kTileQ);
      __syncwarp();
      if (lane < pieces) tma_load_3d(smem_u32(smem + lane * L::kTileQ), &map_q, smem_u32(bar_q), 0, qs + q0, h * p.k_subs + lane * kAtPiece);
    }
    if (!PIECES && lane == 0) {
      mbar_expect_tx(smem_u32(bar_q), (two ? 2 : 1) * L::kTileQ);
      for (int q = 0; q < (two ? 2 : 1); ++q)
        if (KM == 3) tma_load_3d(smem_u32(smem + q * L::kTileQ), &map_q, smem_u32(bar_q), 0, qs + q0 + q * kAtBM, h * p.k_subs);
        else for (int c = 0; c < SUBK; ++c)
          tma_load_2d(smem_u32(smem + q * L::kTileQ + c * (kAtBM * 128)), &map_q, smem_u32(bar_q), h * p.dk + c * 64, qs + q0 + q * kAtBM);
    }
    const int box_rows = p.page_size < kAtBN ? p.page_size : kAtBN;  // page_size is 32, 64 or 128
    int issued = 0, issued_k[2] = {0, 0};  // key tiles; pieces of key tiles (SPLIT: of either group, which has half of the ring)
    constexpr int NSK = SPLIT ? NS / 2 : NS;
    bool ok = true;
    for (int t = 0; t < n_tiles; ++t, ++issued) {
      const int s = t % NS;
      const int kt = tile_at(t);
      if constexpr (PIECES) {  // the pieces of the tile's key rows (SPLIT: of two tiles in turn), then its values
        if (!SPLIT || (t & 1) == 0) {
          const int n_q = SPLIT && t + 1 < n_tiles ? 2 : 1;
          for (int i = 0; ok && i < pieces * n_q; ++i) {
            const int pc = i / n_q, q = i % n_q, n = q == 0 ? issued_k[0] : issued_k[1];
            const int st = q * NSK + n % NSK;
            if (n >= NSK) ok = mbar_wait(smem_u32(&bar_k_empty[st]), ((n / NSK) - 1) & 1, abort_flag, p.status);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            if (lane == 0) mbar_expect_tx(smem_u32(&bar_k_full[st]), L::kTileK);
            __syncwarp();
            uint8_t* dst = smem + L::kOffK + st * L::kTileK;
            if (lane == 0) tma_load_3d(smem_u32(dst + L::kOffKeys), &map_k, smem_u32(&bar_k_full[st]), 0, p.kv_row0[seq] + (kt + q) * kAtBN, pc * kAtPiece);
            if (KM == 2 && lane == 1) tma_load_3d(smem_u32(dst), &map_q, smem_u32(&bar_k_full[st]), 0, qs + q0, h * p.k_subs + pc * kAtPiece);
            if (q == 0) ++issued_k[0];
            else ++issued_k[1];
          }
          if (!ok) break;
        }
        const int sv = t % NSV;
        if (t >= NSV) ok = mbar_wait(smem_u32(&bar_v_empty[sv]), ((t / NSV) - 1) & 1, abort_flag, p.status);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (lane == 0) mbar_expect_tx(smem_u32(&bar_v_full[sv]), L::kTileV);
        __syncwarp();
        if (lane < SUBV)
          tma_load_2d(smem_u32(smem + L::kOffV + sv * L::kTileV + lane * (kAtBN * 128)), &map_v, smem_u32(&bar_v_full[sv]), kvh * p.dv + lane * 64,
                      p.kv_row0[seq] + kt * kAtBN);
        continue;
      }
      for (int kv = 0; kv < 2; ++kv) {
        uint64_t* full = kv == 0 ? &bar_k_full[s] : &bar_v_full[s];
        uint64_t* empty = kv == 0 ? &bar_k_empty[s] : &bar_v_empty[s];
        if (t >= NS) ok = mbar_wait(smem_u32(empty), ((t / NS) - 1) & 1, abort_flag, p.status);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (lane == 0) mbar_expect_tx(smem_u32(full), kv == 0 ? L::kTileK : L::kTileV);
        __syncwarp();
        uint8_t* dst = smem + (kv == 0 ? L::kOffK + s * L::kTileK : L::kOffV + s * L::kTileV);
        const int sub = kv == 0 ? SUBK : SUBV;
        if constexpr (KM == 3) {
          const int row = p.kv_row0[seq] + kt * kAtBN;
          if (kv == 0 && lane == 0) tma_load_3d(smem_u32(dst), &map_k, smem_u32(full), 0, row, 0);
          if (kv == 1 && lane < SUBV) tma_load_2d(smem_u32(dst + lane * (kAtBN * 128)), &map_v, smem_u32(full), kvh * p.dv + lane * 64, row);
          continue;
        }
        if constexpr (LATENT) {
          // rows behind the sequence's last key belong to the next sequence, or lie outside the buffer and arrive as zeros
          const int row = p.kv_row0[seq] + kt * kAtBN;
          for (int c = lane; c < sub; c += 32) {
            const bool shared_part = kv == 0 && c >= p.kn_blocks;
            const int x = shared_part ? (c - p.kn_blocks) * 64 : (kv == 0 ? h * p.kn_blocks + c : h * SUBV + c) * 64;
            tma_load_2d(smem_u32(dst + c * (kAtBN * 128)), shared_part ? &map_r : (kv == 0 ? &map_k : &map_v), smem_u32(full), x, row);
          }
          continue;
        }
        const int n_copy = (kAtBN / box_rows) * sub;
        for (int i = lane; i < n_copy; i += 32) {
          const int pg = i / sub, c = i - pg * sub;
          const int key0 = kt * kAtBN + pg * box_rows;
          // pages past the context are never read by an unmasked score; the scratch page 0 keeps the copy inside the cache
          const int page = key0 < ctx ? p.block_tables[static_cast<long long>(seq) * p.bt_stride + key0 / p.page_size] : 0;
          const int row = (page * p.KV + kvh) * p.page_size + (key0 % p.page_size);
          const uint32_t off = c * (kAtBN * 128) + pg * box_rows * 128;
          tma_load_2d(smem_u32(dst + off), kv == 0 ? &map_k : &map_v, smem_u32(full), c * 64, row);
        }
      }
      if (!ok) break;
    }
    if (lane == 0 && *abort_flag) {
      // a wait ran out somewhere in the CTA: before shared memory goes away let the copies already issued land (bounded)
      for (int q = 0; PIECES && q < 2; ++q)
        for (int n = issued_k[q] > NSK ? issued_k[q] - NSK : 0; n < issued_k[q]; ++n) {
          const unsigned long long t0 = globaltimer_ns();
          while (!mbar_try_wait(smem_u32(&bar_k_full[q * NSK + n % NSK]), (n / NSK) & 1) && globaltimer_ns() - t0 < 20000000ull) {
          }
        }
      for (int t = issued > NSV ? issued - NSV : 0; PIECES && t < issued; ++t) {
        const unsigned long long t0 = globaltimer_ns();
        while (!mbar_try_wait(smem_u32(&bar_v_full[t % NSV]), (t / NSV) & 1) && globaltimer_ns() - t0 < 20000000ull) {
        }
      }
      for (int t = issued > NS ? issued - NS : 0; !PIECES && t < issued; ++t) {
        const unsigned long long t0 = globaltimer_ns();
        while (!(mbar_try_wait(smem_u32(&bar_k_full[t % NS]), (t / NS) & 1) && mbar_try_wait(smem_u32(&bar_v_full[t % NS]), (t / NS) & 1)) &&
               globaltimer_ns() - t0 < 20000000ull) {
        }
      }
    }
    __syncwarp();
  } else if (warp == kIssuer || warp == kIssuerPV || (SPLIT && warp == kIssuer2)) {
    // ---------------- MMA issuers ----------------
    // Work items (key tile j, query tile q) in order: (j, 0), (j, 1) for every j the query tile sees. Each query tile has two score
    // slots, used by its key tiles in turn.
    // A tcgen05.mma holds the issuing thread until the tensor pipe accepts it and the pipe queues next to nothing, so the pipe idles
    // whenever its issuer does anything else, and even a wait on a barrier that is already complete costs a few hundred cycles.
    // Hence two issuing threads with loops of their own: one thread of warp 0 issues the Q K^T of every item as soon as its slot is
    // free again (the P V that read the probabilities kept there has retired) and its K tile has landed; one thread of warp 2
    // issues the P V of every item once its probabilities are written and its V tile has landed. While one of them waits, the other
    // feeds the pipe. Everything the two depend on travels through mbarriers; tcgen05.commit covers the MMAs of its own thread.
    constexpr uint32_t idesc_s = umma_idesc_bf16(kAtBM, kAtBN);
    constexpr uint32_t idesc_o = umma_idesc_bf16_bmn(kAtBM, DV);
    auto valid = [&](int u, int q) {
      if (SPLIT) return (u & 1) == q;
      const int j = tile_at(u);
      return q == 0 ? ((j >= a0 || j < kept_tiles) && j < b0) : ((j >= a1 || j < kept_tiles) && j < b1);
    };
    auto advance = [&](int& u, int& q) {  // next valid item (u: place in the CTA's tile list); u == n_tiles when there is none
      do {
        if (two && q == 0) q = 1;
        else { q = 0; ++u; }
      } while (u < n_tiles && !valid(u, q));
    };
    auto last_of_tile = [&](int u, int q) { return SPLIT || !two || q == 1 || !valid(u, 1); };
    // key tiles of query tile q before tile j (the same count its softmax warps keep)
    auto count_at = [&](int u, int q) {
      if (SPLIT) return u >> 1;
      const int j = tile_at(u), a = q == 0 ? a0 : a1;
      return j < kept_tiles ? j : j - max(a, kept_tiles) + kept_tiles;
    };
    if (lane == 0) {
      bool ok = true;
      int u = 0, q = 0;
      if (n_tiles > 0 && !valid(u, q)) advance(u, q);
      if (warp != kIssuerPV) {
        if (KM != 2) ok = mbar_wait(smem_u32(bar_q), 0, abort_flag, p.status);
        if (warp == kIssuer2) {
          u = 1;
          q = 1;
        }
        constexpr int NSK = SPLIT ? NS / 2 : NS;
        int piece = 0;  // pieces of this thread's key tiles so far
        const uint64_t desc_q0 = umma_desc_k_sw128(smem_u32(smem)), desc_k0 = umma_desc_k_sw128(smem_u32(smem + L::kOffK));
        int k_seen = -1;  // key tiles whose K has been waited for
        while (ok && u < n_tiles) {
          const int t = count_at(u, q);
          const int s = u % NS;
          const uint32_t slot = q * 2 + (t & 1);
          if (t >= 2) ok = mbar_wait(smem_u32(&bar_pv_done[slot]), ((t >> 1) - 1) & 1, abort_flag, p.status);
          if constexpr (PIECES) {
            const uint32_t d_w = tmem_base + kColS + slot * kAtBN;
            for (int pc = 0; ok && pc < pieces; ++pc, ++piece) {
              const int st = (SPLIT ? q * NSK : 0) + piece % NSK;
              ok = mbar_wait(smem_u32(&bar_k_full[st]), (piece / NSK) & 1, abort_flag, p.status);
              if (!ok) break;
              tc_fence_after();
              const uint64_t desc_q = umma_desc_k_sw128(smem_u32(smem + (KM == 1 ? pc * L::kTileQ : L::kOffK + st * L::kTileK)));
              const uint64_t desc_k = umma_desc_k_sw128(smem_u32(smem + L::kOffK + st * L::kTileK + L::kOffKeys));
              const int subs = min(kAtPiece, p.k_subs - pc * kAtPiece);
              for (int c = 0; c < subs; ++c)
#pragma unroll
                for (int k16 = 0; k16 < 4; ++k16)
                  umma_bf16(d_w, desc_q + static_cast<uint64_t>((c * (kAtBM * 128) + k16 * 32) >> 4), desc_k + static_cast<uint64_t>((c * (kAtBN * 128) + k16 * 32) >> 4),
                            idesc_s, (pc > 0 || c > 0 || k16 > 0) ? 1u : 0u);
              umma_commit(smem_u32(&bar_k_empty[st]));
            }
            if (!ok) break;
            umma_commit(smem_u32(&bar_s_full[slot]));
            if (SPLIT) u += 2;
            else advance(u, q);
            continue;
          }
          if (ok && u > k_seen) {
            ok = mbar_wait(smem_u32(&bar_k_full[s]), (u / NS) & 1, abort_flag, p.status);
            k_seen = u;
          }
          if (!ok) break;
          tc_fence_after();
          const uint64_t desc_q = desc_q0 + static_cast<uint64_t>((q * L::kTileQ) >> 4);
          const uint64_t desc_k = desc_k0 + static_cast<uint64_t>((s * L::kTileK) >> 4);
          const uint32_t d_s = tmem_base + kColS + slot * kAtBN;
#pragma unroll
          for (int k16 = 0; k16 < DK / 16; ++k16) {
            const uint64_t adv_q = static_cast<uint64_t>(((k16 >> 2) * (kAtBM * 128) + (k16 & 3) * 32) >> 4);
            const uint64_t adv_k = static_cast<uint64_t>(((k16 >> 2) * (kAtBN * 128) + (k16 & 3) * 32) >> 4);
            umma_bf16(d_s, desc_q + adv_q, desc_k + adv_k, idesc_s, k16 > 0 ? 1u : 0u);
          }
          if (last_of_tile(u, q)) umma_commit(smem_u32(&bar_k_empty[s]));
          umma_commit(smem_u32(&bar_s_full[slot]));
          advance(u, q);
        }
      } else {
        const uint32_t v_base = smem_u32(smem + L::kOffV);
        while (ok && u < n_tiles) {
          const int t = count_at(u, q);
          const int s = u % NSV;
          const uint32_t slot = q * 2 + (t & 1);
          ok = mbar_wait(smem_u32(&bar_p_full[slot]), (t >> 1) & 1, abort_flag, p.status) &&
               mbar_wait(smem_u32(&bar_v_full[s]), (u / NSV) & 1, abort_flag, p.status);
          if (!ok) break;
          tc_fence_after();
          const uint32_t tmem_p = tmem_base + kColS + slot * kAtBN, d_o = tmem_base + kColO + q * DV;
          const uint64_t desc_v0 = umma_desc_mn_sw128(v_base + s * L::kTileV, kAtBN * 128, 1024);
#pragma unroll
          for (int k16 = 0; k16 < kAtBN / 16; ++k16) {
            // 16 keys = two 8-row swizzle atoms (2048 bytes) further down the V tile; the 64-column blocks of D are kAtBN * 128 bytes apart
            umma_bf16_ts(d_o, tmem_p + k16 * 8, desc_v0 + static_cast<uint64_t>((k16 * 2048) >> 4), idesc_o, (t == 0 && k16 == 0) ? 0u : 1u);
          }
          if (last_of_tile(u, q)) umma_commit(smem_u32(&bar_v_empty[s]));
          umma_commit(smem_u32(&bar_pv_done[slot]));
          advance(u, q);
          if (u >= n_tiles) umma_commit(smem_u32(bar_o_final));
        }
        if (n_tiles == 0) umma_commit(smem_u32(bar_o_final));
      }
      if (!ok) {
        // a wait ran out: let this thread's outstanding MMAs retire (bounded) before tensor memory is released
        uint64_t* drain = &bar_drain[warp == kIssuer ? 0 : (warp == kIssuerPV ? 1 : 2)];
        umma_commit(smem_u32(drain));
        const unsigned long long t0 = globaltimer_ns();
        while (!mbar_try_wait(smem_u32(drain), 0) && globaltimer_ns() - t0 < 20000000ull) {
        }
      }
    }
    __syncwarp();
  } else if (warp >= 4 && (warp < 8 || two)) {
    // ---------------- softmax warps: thread = query row ----------------
    const int q = (warp >> 2) - 1;  // query tile of this warpgroup
    const int r = (warp & 3) * 32 + lane;
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    const int my_rows = q == 0 ? rows_q[0] : rows_q[1], my_first = q == 0 ? first_q[0] : first_q[1];
    const int ja = q == 0 ? a0 : a1, jb = q == 0 ? b0 : b1;
    // this query tile's key tiles: [0, my_kept), then [ja, jb) (SPLIT: every other one)
    const int my_kept = min(kept_tiles, ja), my_tiles = SPLIT ? (n_tiles - q + 1) / 2 : my_kept + jb - ja;
    const int my_pos = my_first + r;
    const float c_log2 = 1.4426950408889634f;
    // scores stay in the units the tensor core delivers; kf turns a difference of scores into a base-2 exponent
    const float kf = p.softcap > 0.f ? c_log2 : p.scale * c_log2;
    float m_run = -INFINITY, l_run = 0.f;
    // gate logits of this row; threads behind the last row read that row's (every branch around tensor-memory accesses stays warp-uniform)
    const int q_rows = SPLIT ? 0 : q * kAtBM;  // rows in front of this group's
    const size_t gate_row = static_cast<size_t>(qs + q0 + q_rows + max(0, min(r, my_rows - 1)));
    const __nv_bfloat16* grow = p.gate != nullptr && !p.gate_heads ? p.gate + gate_row * p.gate_pitch + static_cast<size_t>(h) * p.dv : nullptr;
    const bool gate_vec = grow != nullptr && (p.dv & 7) == 0;  // (then rows, heads and the gate are 16-byte aligned)
    if (grow != nullptr)
      for (int c = 0; c < p.dv; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(grow + c));
    bool ok = true;
    for (int t = 0; t < my_tiles && ok; ++t) {
      const int j = SPLIT ? lo + 2 * t + q : (t < my_kept ? t : ja + t - my_kept);
      const uint32_t slot = q * 2 + (t & 1);
      const uint32_t sb = lane_addr + kColS + slot * kAtBN;
      // warp-uniform: the loop holds warp-collective TMEM accesses
      ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bar_s_full[slot]), (t >> 1) & 1, abort_flag, p.status));
      if (!ok) break;
      tc_fence_after();
      const int key_base = j * kAtBN;
      float f[kAtBN];
      {
        uint32_t* u = reinterpret_cast<uint32_t*>(f);
#pragma unroll
        for (int c = 0; c < kAtBN / 32; ++c) tmem_ld_x32(sb + c * 32, u + c * 32);
        tmem_ld_wait();
      }
      if (p.softcap > 0.f) {
        softcap_tile(f, p.scale / p.softcap, p.softcap);
      }
      // is the whole tile visible to all 128 rows? (row 0 sees the fewest late keys, row 127 the fewest early ones)
      const bool full = key_base + kAtBN <= min(ctx, p.causal ? my_first + 1 : ctx) && (p.window <= 0 || key_base >= my_first + kAtBM - p.window || key_base + kAtBN <= p.keep_first) && my_rows == kAtBM;
      if (!full) {
        // visible keys of this row inside the tile: [vlo, vhi)
        int vhi = min(ctx, p.causal ? my_pos + 1 : ctx) - key_base;
        int vlo = (p.window > 0 ? max(0, my_pos - p.window + 1) : 0) - key_base;
        if (r >= my_rows) vhi = vlo = 0;
        const int kept = p.keep_first - key_base;  // keys of the tile in front of this one stay visible
#pragma unroll
        for (int i = 0; i < kAtBN; ++i) f[i] = ((i >= vlo || i < kept) && i < vhi) ? f[i] : -INFINITY;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < kAtBN; i += 8) {
        mx4[0] = fmax3(mx4[0], f[i], f[i + 1]);
        mx4[1] = fmax3(mx4[1], f[i + 2], f[i + 3]);
        mx4[2] = fmax3(mx4[2], f[i + 4], f[i + 5]);
        mx4[3] = fmax3(mx4[3], f[i + 6], f[i + 7]);
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // The running maximum only follows the scores when one of the warp's rows has outgrown it by more than 2^8: a stale
      // maximum costs nothing but head-room (probabilities up to 256), a new one costs a pass over the O accumulator.
      float m_new = m_run;
      if (t == 0) {
        m_new = mx;
      } else if (__any_sync(0xffffffffu, (mx - m_run) * kf > 8.f)) {
        m_new = fmaxf(m_run, mx);
        const float alpha = m_new == -INFINITY ? 1.f : ex2_approx((m_run - m_new) * kf);
        // P V of the previous key tile must have retired before the accumulator is touched (these scores were issued ahead of it)
        ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bar_pv_done[q * 2 + ((t - 1) & 1)]), ((t - 1) >> 1) & 1, abort_flag, p.status));
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int c0 = 0; c0 < DV; c0 += 32) {
          uint32_t v[32];
          tmem_ld_x32(lane_addr + kColO + q * DV + c0, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
          tmem_st_x32(lane_addr + kColO + q * DV + c0, v);
        }
        l_run *= alpha;
      }
      m_run = m_new;
      const float neg_mk = m_new == -INFINITY ? 0.f : -m_new * kf;
      // probabilities -> packed bf16 over the first half of the score slot's columns (every score is in registers by now)
      float ls4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < kAtBN / 32; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float p0 = ex2_approx(fmaf(f[c * 32 + i], kf, neg_mk)), p1 = ex2_approx(fmaf(f[c * 32 + i + 1], kf, neg_mk));
          const float p2 = ex2_approx(fmaf(f[c * 32 + i + 2], kf, neg_mk)), p3 = ex2_approx(fmaf(f[c * 32 + i + 3], kf, neg_mk));
          ls4[0] += p0;
          ls4[1] += p1;
          ls4[2] += p2;
          ls4[3] += p3;
          pk[i >> 1] = pack_bf162(p0, p1);
          pk[(i >> 1) + 1] = pack_bf162(p2, p3);
        }
        tmem_st_x16(sb + c * 16, pk);
      }
      l_run += (ls4[0] + ls4[1]) + (ls4[2] + ls4[3]);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&bar_p_full[slot]));
    }
    // ---------------- epilogue ----------------
    if (ok) ok = mbar_wait(smem_u32(bar_o_final), 0, abort_flag, p.status);
    ok = __all_sync(0xffffffffu, ok && *abort_flag == 0);
    if constexpr (SPLIT) {
      if (ok) {  // every copy has landed and every MMA has retired: the maxima and sums pass through the key stages
        float* ml = reinterpret_cast<float*>(smem + L::kOffK) + q * 256;
        ml[r] = m_run;
        ml[128 + r] = l_run;
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(bar_ml));
        ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(bar_ml), 0, abort_flag, p.status));
      }
    }
    if (ok) {
      tc_fence_after();
      float w_mine = 1.f, w_other = 0.f;  // SPLIT: weights of this group's and the other one's accumulator
      if constexpr (SPLIT) {
        const float* ml = reinterpret_cast<const float*>(smem + L::kOffK) + (1 - q) * 256;
        const float m2 = ml[r], l2 = ml[128 + r], m = fmaxf(m_run, m2);
        w_mine = m_run == -INFINITY ? 0.f : ex2_approx((m_run - m) * kf);
        w_other = m2 == -INFINITY ? 0.f : ex2_approx((m2 - m) * kf);
        l_run = l_run * w_mine + l2 * w_other;
        m_run = m;
      }
      if (p.sink != nullptr) l_run += ex2_approx(p.sink[h] * c_log2 - m_run * kf);  // relative to the running maximum
      float inv = l_run > 0.f ? p.out_mult / l_run : 0.f;
      const size_t trow = static_cast<size_t>(qs + q0 + q_rows + r);
      __nv_bfloat16* orow = p.out + trow * p.out_pitch + static_cast<size_t>(h) * p.dv;
      if (!LATENT && p.gate_heads) inv /= 1.f + __expf(-bf2f(p.gate[gate_row * p.gate_pitch + h]));
      // SPLIT: each group stores half of the columns, from both accumulators
      const int c_first = SPLIT ? q * (DV / 2) : 0, c_last = SPLIT ? c_first + DV / 2 : DV;
#pragma unroll 1
      for (int c0 = c_first; c0 < c_last; c0 += 32) {
        uint4 gv[4];  // the gate logits of this step, all on their way before the first is used
        if (gate_vec) {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (c0 + i * 8 < p.dv) gv[i] = *reinterpret_cast<const uint4*>(grow + c0 + i * 8);
        }
        uint32_t v[32];
        if (my_tiles > 0) {
          tmem_ld_x32(lane_addr + kColO + q * DV + c0, v);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = 0u;
        }
        if constexpr (SPLIT) {
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * w_mine);
          if (n_tiles > 1 - q) {  // the other group has had a tile
            uint32_t v2[32];
            tmem_ld_x32(lane_addr + kColO + (1 - q) * DV + c0, v2);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) + __uint_as_float(v2[i]) * w_other);
          }
        }
        if (LATENT) {
          if (r < my_rows) {
            const bool vec = (p.dv & 7) == 0;  // (then rows, heads and the gate are 16-byte aligned as well)
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              if (c0 + i >= p.dv) break;
              float w[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) w[e] = __uint_as_float(v[i + e]) * inv;
              if (vec) {
                if (grow != nullptr) gate8(w, gv[i / 8]);
                *reinterpret_cast<uint4*>(orow + c0 + i) =
                    make_uint4(pack_bf162(w[0], w[1]), pack_bf162(w[2], w[3]), pack_bf162(w[4], w[5]), pack_bf162(w[6], w[7]));
              } else {
#pragma unroll
                for (int e = 0; e < 8; ++e)
                  if (c0 + i + e < p.dv) orow[c0 + i + e] = f2bf(grow != nullptr ? w[e] / (1.f + __expf(-bf2f(grow[c0 + i + e]))) : w[e]);
              }
            }
          }
        } else if (r < my_rows) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c0 + i >= p.dv) break;
            float w[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) w[e] = __uint_as_float(v[i + e]) * inv;
            if (grow != nullptr) gate8(w, gv[i / 8]);
            *reinterpret_cast<uint4*>(orow + c0 + i) = make_uint4(pack_bf162(w[0], w[1]), pack_bf162(w[2], w[3]), pack_bf162(w[4], w[5]), pack_bf162(w[6], w[7]));
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kIssuer) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

template <int DK, int DV, int QT, bool LATENT, int KM = 0>
static int launch_prefill_tc_maps(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mr, const AttnTcParams& p,
                                  int num_tiles, cudaStream_t st) {
  using L = typename AttnTcLayout<DK, DV, QT, KM>::T;
  static PerDeviceOnce attr_once;
  if (attr_once.first()) {
    cudaError_t e = cudaFuncSetAttribute(prefill_attn_tc_kernel<DK, DV, QT, LATENT, KM>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kBytes);
    if (e != cudaSuccess) throw std::runtime_error(std::string("prefill attention (tcgen05): cudaFuncSetAttribute: ") + cudaGetErrorString(e));
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(num_tiles, p.H);
  cfg.blockDim = dim3(L::kThreads);
  cfg.dynamicSmemBytes = L::kBytes;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = g_pdl_enabled ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  cudaError_t e = cudaLaunchKernelEx(&cfg, prefill_attn_tc_kernel<DK, DV, QT, LATENT, KM>, mq, mk, mv, mr, p);
  if (e != cudaSuccess) throw std::runtime_error(std::string("prefill attention (tcgen05) launch: ") + cudaGetErrorString(e));
  return 0;
}

template <int DK, int DV, int QT>
static int launch_prefill_tc_t(const void* q, long long q_stride, long long T, const void* kc, const void* vc, long long cache_rows, const AttnTcParams& p,
                               int num_tiles, cudaStream_t st) {
  CUtensorMap mq, mk, mv;
  encode_map_2d(&mq, 0, q, static_cast<uint64_t>(T), static_cast<uint64_t>(p.H) * p.dk, static_cast<uint64_t>(q_stride) * 2, kAtBM, 64, 128);
  const uint32_t box_rows = p.page_size < kAtBN ? p.page_size : kAtBN;
  encode_map_2d(&mk, 0, kc, static_cast<uint64_t>(cache_rows), p.dk, static_cast<uint64_t>(p.dk) * 2, box_rows, 64, 128);
  encode_map_2d(&mv, 0, vc, static_cast<uint64_t>(cache_rows), p.dv, static_cast<uint64_t>(p.dv) * 2, box_rows, 64, 128);
  return launch_prefill_tc_maps<DK, DV, QT, false>(mq, mk, mv, mv, p, num_tiles, st);
}

// ---- latent layout -----------------------------------------------------------------------------------------------------
// Operand widths the kernel is instantiated for: the value columns of a head are padded to the returned width (0: not available,
// dk = 64-padded unrotated + rotated columns must be one of 128, 192, 256 and dv at most 256).
int prefill_latent_tc_dv(int dk, int dv) {
  if (dk != 128 && dk != 192 && dk != 256) return 0;
  if (dv <= 64 && dk == 128) return 64;
  if (dv <= 128) return 128;
  if (dv <= 256 && dk == 256) return 256;
  return 0;
}
int prefill_latent_tc_tile_rows(int dv_padded) { return dv_padded <= 128 ? 256 : 128; }

int launch_prefill_latent_tc(const LatentTcArgs& a, cudaStream_t st) {
  if (a.num_tiles == 0) return 0;
  const int DV = prefill_latent_tc_dv(a.dk, a.dv);
  if (DV == 0 || a.kn % 64 != 0 || a.kn <= 0 || a.kn >= a.dk) return 1;
  AttnTcParams p = {};
  p.q_start = a.q_start;
  p.q_len = a.q_len;
  p.ctx_lens = a.ctx;
  p.tile_seq = a.tile_seq;
  p.tile_q0 = a.tile_q0;
  p.out = static_cast<__nv_bfloat16*>(a.out);
  p.H = p.KV = a.H;
  p.page_size = kAtBN;
  p.scale = a.scale;
  p.window = a.window;
  p.causal = 1;
  p.status = a.status;
  p.dk = a.dk;
  p.kv_row0 = a.kv_row0;
  p.kn_blocks = a.kn / 64;
  p.dv = a.dv;
  p.out_pitch = a.out_pitch;
  p.gate = static_cast<const __nv_bfloat16*>(a.gate);
  p.gate_pitch = a.gate_pitch;
  p.sink = a.sink;
  p.out_mult = 1.f;
  CUtensorMap mq, mk, mv, mr;
  const uint64_t H = static_cast<uint64_t>(a.H), rows = static_cast<uint64_t>(a.kv_rows);
  encode_map_2d(&mq, 0, a.q, static_cast<uint64_t>(a.T), H * a.dk, static_cast<uint64_t>(a.q_pitch) * 2, kAtBM, 64, 128);
  encode_map_2d(&mk, 0, a.k, rows, H * a.kn, static_cast<uint64_t>(a.kv_pitch) * 2, kAtBN, 64, 128);
  encode_map_2d(&mv, 0, a.v, rows, H * DV, static_cast<uint64_t>(a.kv_pitch) * 2, kAtBN, 64, 128);
  encode_map_2d(&mr, 0, a.kr, rows, static_cast<uint64_t>(a.dk - a.kn), static_cast<uint64_t>(a.kr_pitch) * 2, kAtBN, 64, 128);
#define DLV_LAT(DKV, DVV, QTV) \
  if (a.dk == DKV && DV == DVV) return launch_prefill_tc_maps<DKV, DVV, QTV, true>(mq, mk, mv, mr, p, a.num_tiles, st)
  DLV_LAT(128, 64, 2);
  DLV_LAT(128, 128, 2);
  DLV_LAT(192, 128, 2);
  DLV_LAT(256, 128, 2);
  DLV_LAT(256, 256, 1);
#undef DLV_LAT
  return 1;
}

// ---- wide rows ---------------------------------------------------------------------------------------------------------
int prefill_attention_wide_tile_rows(int k_width, int dv) {
  if (k_width <= 0 || dv <= 0 || k_width % 8 != 0 || dv % 8 != 0 || dv > 256) return 0;
  return k_width > 256 || dv > 128 ? kAtBM : 2 * kAtBM;
}

template <int DK, int DV, int QT, int KM>
static int launch_wide_t(const WideTcArgs& a, const AttnTcParams& p, cudaStream_t st) {
  CUtensorMap mq, mk, mv;
  const uint64_t width = static_cast<uint64_t>(p.k_subs) * 64, rows = static_cast<uint64_t>(a.kv_rows), v_width = static_cast<uint64_t>(p.KV) * p.dv;
  const uint32_t blocks = KM == 3 ? DK / 64 : kAtPiece;
  encode_map_kchunks(&mq, a.q, static_cast<uint64_t>(a.T), p.H * width, p.H * width * 2, kAtBM, blocks);
  encode_map_kchunks(&mk, a.k, rows, width, width * 2, kAtBN, blocks);
  encode_map_2d(&mv, 0, a.v, rows, v_width, v_width * 2, kAtBN, 64, 128);
  return launch_prefill_tc_maps<DK, DV, QT, false, KM>(mq, mk, mv, mv, p, a.num_tiles, st);
}

int launch_prefill_wide_tc(const WideTcArgs& a, AttnExtra x, cudaStream_t st) {
  if (a.num_tiles == 0) return 0;
  const int subs = (a.k_width + 63) / 64;
  if (prefill_attention_wide_tile_rows(a.k_width, a.dv) == 0 || x.keep_first != 0 || x.sink != nullptr) return 1;
  AttnTcParams p = {};
  p.q_start = a.q_start;
  p.q_len = a.q_len;
  p.ctx_lens = a.ctx;
  p.tile_seq = a.tile_seq;
  p.tile_q0 = a.tile_q0;
  p.kv_row0 = a.kv_row0;
  p.out = static_cast<__nv_bfloat16*>(a.out);
  p.H = a.H;
  p.KV = a.KV;
  p.page_size = kAtBN;
  p.scale = a.scale;
  p.window = a.window;
  p.causal = 1;
  p.dk = subs * 64;
  p.dv = a.dv;
  p.k_subs = subs;
  p.gate = static_cast<const __nv_bfloat16*>(x.gate);
  p.gate_pitch = x.gate_pitch;
  p.gate_heads = x.gate_heads;
  p.out_mult = x.out_mult;
  p.out_pitch = x.out_pitch > 0 ? x.out_pitch : static_cast<long long>(a.H) * a.dv;
  p.status = a.status;
  if (subs <= 4) {
    if (a.dv <= 64) {
      if (subs <= 2) return launch_wide_t<128, 64, 2, 3>(a, p, st);
      return subs <= 3 ? launch_wide_t<192, 64, 2, 3>(a, p, st) : launch_wide_t<256, 64, 2, 3>(a, p, st);
    }
    if (a.dv <= 128) {
      if (subs <= 2) return launch_wide_t<128, 128, 2, 3>(a, p, st);
      return subs <= 3 ? launch_wide_t<192, 128, 2, 3>(a, p, st) : launch_wide_t<256, 128, 2, 3>(a, p, st);
    }
    return launch_wide_t<256, 256, 1, 3>(a, p, st);
  }
#define DLV_WIDE(DVV, QTV) return subs <= kAtResident ? launch_wide_t<0, DVV, QTV, 1>(a, p, st) : launch_wide_t<0, DVV, QTV, 2>(a, p, st)
  if (a.dv <= 64) DLV_WIDE(64, 2);
  if (a.dv <= 128) DLV_WIDE(128, 2);
  DLV_WIDE(256, 1);
#undef DLV_WIDE
}

// Query rows one CTA of the tcgen05 prefill kernel covers: two 128-row tiles share the K / V tiles where their two accumulators fit
// tensor memory beside the two score slots.
int prefill_attention_tc_tile_rows(int D) { return D <= 128 ? 256 : 128; }

// tile arrays: prefill_attention_tc_tile_rows(max(dk, dv)) query rows per tile. page_size must be 32, 64 or 128. Returns 1 for an unsupported
// head size (multiples of 8 up to 256) or page size.
int launch_prefill_attention_tc(const void* q, long long q_stride, long long T, const void* kc, const void* vc, long long num_pages, const int* bt,
                                int bt_stride, const int* q_start, const int* q_len, const int* ctx, const int* tile_seq, const int* tile_q0,
                                int num_tiles, void* out, int H, int KV, int dk, int dv, int page, float scale, float cap, int window, int causal,
                                AttnExtra x, int* status, cudaStream_t st) {
  if (num_tiles == 0) return 0;
  const int D = dk > dv ? dk : dv;
  if ((page != 32 && page != 64 && page != 128) || dk % 8 != 0 || dv % 8 != 0 || dk <= 0 || dv <= 0 || D > 256) return 1;
  AttnTcParams p = {};
  p.block_tables = bt;
  p.bt_stride = bt_stride;
  p.q_start = q_start;
  p.q_len = q_len;
  p.ctx_lens = ctx;
  p.tile_seq = tile_seq;
  p.tile_q0 = tile_q0;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.H = H;
  p.KV = KV;
  p.page_size = page;
  p.scale = scale;
  p.softcap = cap;
  p.window = window;
  p.causal = causal;
  p.keep_first = window > 0 ? x.keep_first : 0;
  p.sink = x.sink;
  p.gate = static_cast<const __nv_bfloat16*>(x.gate);
  p.gate_pitch = x.gate_pitch;
  p.gate_heads = x.gate_heads;
  p.out_mult = x.out_mult;
  p.dk = dk;
  p.dv = dv;
  p.out_pitch = x.out_pitch > 0 ? x.out_pitch : static_cast<long long>(H) * dv;
  p.status = status;
  const long long cache_rows = num_pages * KV * page;
  if (D <= 64) return launch_prefill_tc_t<64, 64, 2>(q, q_stride, T, kc, vc, cache_rows, p, num_tiles, st);
  if (D <= 128 && dv <= 64) return launch_prefill_tc_t<128, 64, 2>(q, q_stride, T, kc, vc, cache_rows, p, num_tiles, st);
  if (D <= 128) return launch_prefill_tc_t<128, 128, 2>(q, q_stride, T, kc, vc, cache_rows, p, num_tiles, st);
  return launch_prefill_tc_t<256, 256, 1>(q, q_stride, T, kc, vc, cache_rows, p, num_tiles, st);
}

}  // namespace dlv
