// C++ interface between the torch bindings and the kernel launchers (no torch types below this line).
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <stddef.h>
#include <stdint.h>

namespace dlv {

// JQ4 weights are held tile-packed on the device: [ceil(N/128)][ceil(K/128)][10240] bytes. One 10240-byte stage holds a
// 128-row x 128-k tile: 8192 bytes of packed nibbles, row r at r*64, its four 16-byte blocks (32 elements each, split-half
// nibble order) stored at chunk position (block ^ ((r >> 1) & 3)), followed by 2048 bytes of fp32 scales [row][4].
// Rows / k beyond N / K are zero (zero scale).
constexpr int kQ4StageBytes = 10240;

struct GemmWeightDesc {
  int N = 0, K = 0;
  bool is_q4 = false;
  const void* data = nullptr;  // bf16 [N, K] or the tile-packed JQ4 bytes
  CUtensorMap map_w;           // dense: [N, K] (3-D chunked form when w3d); JQ4: the packed stages as rows of 1 KB
  bool w3d = false;
};

// Peer-memory state of the fused GEMM + all-reduce epilogue (all pointers are device addresses mapped in this process).
struct GemmTpArgs {
  int size = 1, rank = 0;
  int ncta_max = 0;              // flag matrix row length
  long long slab = 0;            // bf16 elements per (parity, source) receive slab
  unsigned long long recv[8];    // receive area of every rank
  unsigned long long flags[8];   // flag matrix of every rank
  unsigned int* rounds = nullptr;  // local [ncta_max]
  unsigned int* call = nullptr;    // local [2]
  long long wait_limit_cycles = 0; // bound of every peer-flag wait in SM cycles (0: the default of about 2 s)
  // What the row-parallel GEMM epilogue does with its partial tile: 0 = store it into every rank's slab, wait for the peers and
  // reduce (GEMM + all-reduce in one kernel); 1 = store it into every rank's slab, publish and leave (launch_tp_reduce_norm waits,
  // sums the ranks and applies the residual add and the norm that follow the projection); 2 = store it into this rank's own slab,
  // publish and leave (the reduce kernel sums through the NVSwitch multicast address mc_recv with multimem.ld_reduce).
  int mode = 0;
  unsigned long long mc_recv = 0;  // multicast (NVLS) address of the receive area, 0 when not bound
  mutable int last_ctas = 0;       // CTAs of the last fused launch (the reduce kernel waits for that many publications per rank)
};

// Peer-memory state of the GEMM -> reduce-scatter -> all-gather path for prefill-size batches (see gemm_tc_run_scatter).
struct GemmScatterArgs {
  int size = 1, rank = 0;
  long long recv_elems = 0;      // capacity of a receive area in bf16 elements: size * rows_per_rank * N must fit
  long long gather_elems = 0;    // capacity of a gather area: M * N must fit
  unsigned long long recv[8];    // every rank's receive area, bf16 [size sources][rows_per_rank][N] for the launch at hand
  unsigned long long gather[8];  // every rank's gather area, bf16 [M][N]: rows arrive reduced from their owners
  unsigned long long flags[8];   // every rank's u32 [24], cumulative: [src] partial tiles from src, [8 + src] reduced row groups from
                                 // src, [16 + src] row groups src pushed for an all-gather -> GEMM
};
// How a launch of M token rows is cut over the ranks: rank r owns rows [r * rows_per_rank, min(M, (r + 1) * rows_per_rank)).
struct GemmScatterPlan {
  int rows_per_rank;  // a multiple of kScatterGroupRows
  int rows[8];        // rows owned per rank (0 for ranks beyond the end)
  int tiles[8];       // GEMM CTAs that publish to rank r, per source rank
  int groups[8];      // reduce CTAs of rank r (kScatterGroupRows rows each)
};
constexpr int kScatterGroupRows = 8;
GemmScatterPlan gemm_scatter_plan(int M, int N, int size);
bool gemm_scatter_supported(const GemmWeightDesc* w, int M, const GemmScatterArgs* a);

void gemm_weight_init(GemmWeightDesc* w);
int gemm_num_sms();
void gemm_set_pdl(bool on);  // programmatic dependent launch of the GEMM kernels (on by default)
void gemm_tc_run(const GemmWeightDesc* w, const void* x, int M, int ldx, void* out, int ldo, bool out_f32, const float* bias,
                 float* ws, size_t ws_floats, int* counters, int n_counters, int* status, int force_splits, cudaStream_t st,
                 const GemmTpArgs* tp = nullptr);
// Grouped (mixture-of-experts) GEMM over rows sorted by expert; `w` stacks the local experts (JQ4: each expert padded to whole
// 128-row tiles), `items` is the device work list of launch_moe_items built with the same token tile `bn`.
// arguments of the q | k | v epilogue (per-head RMSNorm, rotary embedding, paged KV write); see gemm_tc_run_qkv
struct GemmQkvArgs {
  const int* positions;        // [M]
  const long long* slots;      // [M] flat cache rows, < 0: skip the cache write
  const void* q_norm_w;        // bf16 [128] or nullptr
  const void* k_norm_w;
  const float* cos_t;          // [max_pos, rot_half] or nullptr
  const float* sin_t;
  void* k_cache;               // bf16 [blocks, KV, block_size, 128]
  void* v_cache;
  int heads, kv_heads, block_size, rot_half, max_pos;
  float eps, norm_offset;
};
void gemm_tc_run_qkv(const GemmWeightDesc* w, const void* x, int M, int ldx, void* q_out, int ldo, const float* bias, const GemmQkvArgs* a,
                     float* ws, size_t ws_floats, int* counters, int n_counters, int* status, cudaStream_t st);
void gemm_tc_run_grouped_act(const GemmWeightDesc* w, int n_per_expert, const void* x, int rows, int ldx, void* out, int ldo,
                             const int* items, int max_items, int bn, int splits, int act, int* status, cudaStream_t st);
// gate | up projection with act(gate) * up computed in the epilogue (weights interleaved per tile; see gemm.cu)
void gemm_tc_run_act(const GemmWeightDesc* w, const void* x, int M, int ldx, void* out, int ldo, int act, float* ws, size_t ws_floats,
                     int* counters, int n_counters, int* status, cudaStream_t st);
void gemm_tc_run_grouped(const GemmWeightDesc* w, int n_per_expert, const void* x, int rows, int ldx, void* out, int ldo,
                         const int* items, int max_items, int bn, int splits, int* status, cudaStream_t st);
// CUDA-core variant for decode-size groups (at most `mt` = 4 or 8 rows per work item; items built with bn == mt)
void gemv_grouped_run(const GemmWeightDesc* w, int n_per_expert, const void* x, int ldx, void* out, int ldo, const int* items,
                      int max_items, int mt, cudaStream_t st);
// row_map / row_div (optional): grouped row r reads x row row_map[r] / row_div (x ungathered, row_map the grouping permutation)
bool gemv_grouped_act_run(const GemmWeightDesc* w, int n_per_expert, const void* x, int ldx, void* out, int ldo, const int* items, int max_items,
                          int act, const int* row_map, int row_div, cudaStream_t st);
// Row-parallel projection whose partial tiles go straight to the rank that owns their token rows (epilogue EPI = 3, no waiting
// inside the GEMM). Follow it with launch_scatter_reduce and launch_scatter_finish on the same stream.
void gemm_tc_run_scatter(const GemmWeightDesc* w, const void* x, int M, int ldx, const GemmScatterArgs* a, int* status, cudaStream_t st);
// all-gather -> GEMM: every rank holds the rows it owns (the cut of gemm_scatter_plan) of the activations [M, K]. launch_gather_push
// copies them into every rank's gather area and publishes one count per CTA; gemm_tc_run_gathered multiplies the local gather
// area by `w`, its activation producers wait per token tile for the owners' counts (group_targets[src], cumulative).
bool gemm_gathered_supported(const GemmWeightDesc* w, int M, const GemmScatterArgs* a);
void launch_gather_push(const GemmScatterArgs* a, const GemmScatterPlan* plan, const void* x_own, int M, int K, int* status, cudaStream_t st);
void gemm_tc_run_gathered(const GemmWeightDesc* w, int M, const GemmScatterArgs* a, const unsigned* group_targets, void* out, int ldo,
                          const float* bias, float* ws, size_t ws_floats, int* counters, int n_counters, int* status, cudaStream_t st);
// true when the fused all-reduce epilogue can take this problem (one wave of CTAs, rows and columns inside the slab)
bool gemm_tp_supported(const GemmWeightDesc* w, int M, const GemmTpArgs* tp);
void gemv_simt_run(const GemmWeightDesc* w, const void* x, int M, int ldx, void* out, int ldo, bool out_f32, const float* bias,
                   cudaStream_t st);

// elementwise.cu
void launch_rmsnorm(const void* x, void* residual, const void* w, void* y, int T, int H, float eps, float offset, float res_mult,
                    cudaStream_t st);
void launch_layernorm(const void* x, const void* w, const void* b, void* y, int T, int H, float eps, cudaStream_t st);
void launch_act_mul(const void* in, void* out, long long T, int I, int act, cudaStream_t st);
void launch_act(const void* in, void* out, long long n, int act, bool is_f32, cudaStream_t st);
void launch_embedding(const void* table, const int* ids, const void* pos_table, const int* pos, const void* type_table,
                      const int* types, void* out, int T, int H, int vocab, float scale, cudaStream_t st);
int launch_rope_kv(void* qkv, const int* positions, const long long* slots, const void* qn, const void* kn, const float* cos_t,
                   const float* sin_t, void* k_cache, void* v_cache, int T, int H, int KV, int D, int block_size, int rot_half,
                   float eps, float norm_offset, int max_pos, cudaStream_t st);

// Options of the attention kernels beyond scale, soft-cap and window: first keys that stay visible beside the window; a score per head
// that takes part in the softmax without a value; an output gate (out = head * out_mult * sigmoid(gate), one logit per column or one per
// head, of the activations' type); the row pitch of the output (0: H * dv).
struct AttnExtra {
  int keep_first = 0;
  const float* sink = nullptr;  // [H]
  const void* gate = nullptr;   // [T, gate_pitch]
  long long gate_pitch = 0;
  int gate_heads = 0;  // 1: one logit per head
  float out_mult = 1.f;
  long long out_pitch = 0;
};

// attention.cu
int launch_decode_attention(const void* q, long long q_stride, const void* kc, const void* vc, const int* bt, int bt_stride,
                            const int* ctx, void* out, float* po, float* pml, int B, int H, int KV, int D, int page, float scale,
                            float cap, int window, int splits, cudaStream_t st);
int launch_decode_attention_impl(const void* q, long long q_stride, const void* kc, const void* vc, const int* bt, int bt_stride,
                                 const int* ctx, void* out, float* po, float* pml, int* arrivals, int B, int H, int KV, int D, int page,
                                 float scale, float cap, int window, int splits, int impl, cudaStream_t st);
// tensor-core decode kernel with separate key and value widths (multiples of 8, at most 256) and any group size; 1: unsupported shape
int launch_decode_attention_mma(const void* q, long long q_stride, const void* kc, const void* vc, const int* bt, int bt_stride, const int* ctx, void* out,
                                float* po, float* pml, int B, int H, int KV, int dk, int dv, int page, float scale, float cap, int window, AttnExtra x,
                                int splits, cudaStream_t st);
// one CTA per (row, query head) on CUDA cores, fp32 or bf16, any width; row_seq: sequence of every row (nullptr: row number)
// wide: queries of dk columns against whole cache rows k [pages, 1, page, dk], values v [pages, 1, page, KV * dv]
int launch_attention_rows(const void* q, long long q_stride, const void* kc, const void* vc, const int* bt, int bt_stride, const int* row_seq,
                          const int* positions, void* out, int T, int H, int KV, int dk, int dv, int page, float scale, float cap, int window, bool wide,
                          AttnExtra x, bool is_f32, cudaStream_t st);
int launch_prefill_attention(const void* q, long long q_stride, const void* kc, const void* vc, const int* bt, int bt_stride,
                             const int* q_start, const int* q_len, const int* ctx, const int* tile_seq, const int* tile_q0,
                             int num_tiles, void* out, int H, int KV, int D, int page, float scale, float cap, int window,
                             int causal, cudaStream_t st);

// attention_tc.cu: tcgen05 / TMA prefill attention; tile arrays hold prefill_attention_tc_tile_rows(D) query rows per tile
int prefill_attention_tc_tile_rows(int D);
extern bool g_gemm_persist;    // gemm_persist.cu: prefill-size JQ4 projections on the persistent kernel (off by default)
extern bool g_gemm_persist_ordered;  // its issuers take turns in k-block order (bit-reproducible; default) or race
bool gemm_persist_supported(const GemmWeightDesc* w, int M, int ldx);
bool gemm_persist_preferred(const GemmWeightDesc* w, int M);
void gemm_persist_run(const GemmWeightDesc* w, const void* x, int M, int ldx, void* out, int ldo, bool out_f32, const float* bias, int* status,
                      cudaStream_t st);
extern bool g_gemm_persist_all;
extern int g_gemm_force_bn;    // gemm.cu: token tile for prefill-size batches (tests, comparisons)
extern int g_gemv_max_rows;     // gemm.cu: most token rows the small-batch GEMV takes (default 8; up to 16)
extern int g_gemv_force_split;  // gemm.cu: warps per CTA of the small-batch GEMV (0: chosen per shape)
extern bool g_gemv_dense;      // gemm.cu: <= 8-row JQ4 projections on the mma.sync GEMV (default on)
bool gemv_dense_supported(const GemmWeightDesc* w, int M, int ldx);
void gemv_dense_run(const GemmWeightDesc* w, const void* x, int M, int ldx, void* out, int ldo, bool out_f32, const float* bias, int act,
                    cudaStream_t st);
extern bool g_gemv_simt_only;  // gemm.cu: grouped JQ4 GEMV on CUDA cores instead of mma.sync (comparisons)
int launch_prefill_attention_tc(const void* q, long long q_stride, long long T, const void* kc, const void* vc, long long num_pages, const int* bt,
                                int bt_stride, const int* q_start, const int* q_len, const int* ctx, const int* tile_seq, const int* tile_q0,
                                int num_tiles, void* out, int H, int KV, int dk, int dv, int page, float scale, float cap, int window, int causal,
                                AttnExtra x, int* status, cudaStream_t st);
// wide rows: query tile height for keys of k_width columns and values of dv columns per head, 0 when the kernel does not take them
int prefill_attention_wide_tile_rows(int k_width, int dv);
// q [T, H * W], gathered keys k [kv_rows, W] (W: k_width padded with zeros to a multiple of 64) and values v [kv_rows, KV * dv]
struct WideTcArgs {
  const void *q, *k, *v;
  long long T, kv_rows;
  int H, KV, k_width, dv;
  const int *q_start, *q_len, *ctx, *kv_row0, *tile_seq, *tile_q0;  // ctx: keys of a sequence in k / v (its query rows are the last q_len)
  int num_tiles;
  void* out;
  float scale;
  int window;
  int* status;
};
int launch_prefill_wide_tc(const WideTcArgs& a, AttnExtra x, cudaStream_t st);

// sampling.cu
void launch_argmax(const float* logits, int ld, int B, int V, const uint32_t* mask, int mask_ld, float softcap, float inv_scale,
                   long long* out_idx, float* out_val, cudaStream_t st);
void launch_logits_post(float* logits, int ld, int B, int V, const uint32_t* mask, int mask_ld, float softcap, float inv_scale,
                        cudaStream_t st);

void launch_sample(const float* logits, int ld, int B, int V, const float* inv_temp, const long long* limits, const float* top_p,
                   const unsigned char* uniform, const float* us, long long* out_tok, int* out_ok, cudaStream_t st);

// exclude-top-choice pick per row (-1: XTC does not apply) and log-probabilities (chosen token + top_n) per row; see sampling.cu
void launch_xtc(const float* logits, int ld, int B, int V, const float* inv_temp, const float* threshold, const unsigned char* fire,
                const int* special, int n_special, long long* out_tok, cudaStream_t st);
void launch_logprobs(const float* logits, int ld, int B, int V, const long long* chosen, int top_n, float* out_chosen, long long* out_idx,
                     float* out_val, cudaStream_t st);

// moe.cu
size_t moe_route_workspace_ints(int T, int E, int k);  // ints of `ws` for the parallel grouping of large batches (0: not needed)
// How experts are chosen and weighted. mode 0: softmax over all, the largest (renorm: divided by their sum); 1: softmax over the k largest logits;
// 2: sigmoid scores, the largest of score + correction among the `keep` best of `groups` equal groups of neighbours (a group counts the sum of
// its two largest choice scores), weights = scores over their sum (+ 1e-20) times scale.
struct MoeRouting {
  int mode = 0, renorm = 0;
  const float* correction = nullptr;  // [E]
  int groups = 1, keep = 1;
  float scale = 1.f;
};
constexpr int kMoeMaxGroups = 64;
void launch_moe_route(const float* logits, int T, int E, int k, const MoeRouting& r, float* w, int* idx, int* counts, int* offsets,
                      int* perm, int* pos, int* ws, cudaStream_t st);
// `range` (optional) = offsets + first local expert and the count of local experts: rows outside
// [offsets[e0], offsets[e0 + ne]) are skipped (expert parallelism: other ranks own them)
void launch_moe_gather(const void* x, const int* perm, int rows, int k, int row_bytes, void* xs, const int* offsets, int e0, int ne,
                       cudaStream_t st);
void launch_moe_combine(const void* ys, const int* pos, const float* w, int T, int k, int H, void* out, const int* offsets, int e0,
                        int ne, cudaStream_t st);
void launch_moe_items(const int* offsets, int e0, int ne, int bn, int max_items, int* items, cudaStream_t st);
bool launch_moe_route_small(const float* logits, int T, int E, int k, const MoeRouting& r, float* w, int* idx, int* counts, int* offsets,
                            int* perm, int* pos, int e0, int ne, int bn, int max_items, int* items, cudaStream_t st);

// comm.cu: fused compute + collective kernels over peer memory (same protocol as the GEMM all-reduce epilogue)
bool comm_rows_supported(const GemmTpArgs* tp, int rows, int H);
void launch_moe_combine_allreduce(const void* ys, const int* pos, const float* w, int T, int k, int H, const int* offsets, int e0, int ne,
                                  void* out, const GemmTpArgs* tp, int* status, cudaStream_t st);
void launch_oneshot_allreduce(const void* x, int rows, int H, void* out, const GemmTpArgs* tp, int* status, cudaStream_t st);
// Second half of a row-parallel projection launched with GemmTpArgs::mode 1 or 2 (see comm.cu): wait for the ranks, sum them, then
// kind 0: out = sum; kind 1: residual += [RMSNorm(post_w)](sum) * res_mult, out = RMSNorm(residual, norm_w). N % 8 == 0, N <= 12288.
void launch_tp_reduce_norm(const GemmTpArgs* tp, int M, int N, int kind, const float* bias, void* residual, const void* post_w, const void* norm_w,
                           void* out, float eps, float offset, float res_mult, int* status, cudaStream_t st);

// Sum the size partial slabs of this rank's rows (+ bias). push: write them to out [M, N] and to every peer's gather area and
// publish (all-reduce, follow with launch_scatter_finish); !push: write them to out [own rows, N] only (reduce-scatter).
// gemm_target: cumulative number of partial tiles every source must have published to this rank.
void launch_scatter_reduce(const GemmScatterArgs* a, const GemmScatterPlan* plan, int M, int N, const float* bias, void* out,
                           unsigned gemm_target, bool push, int* status, cudaStream_t st);
// Wait for the other ranks' reduced rows and copy them from the gather area into out. group_targets[src]: cumulative row groups.
void launch_scatter_finish(const GemmScatterArgs* a, const GemmScatterPlan* plan, int M, int N, void* out, const unsigned* group_targets,
                           int* status, cudaStream_t st);

struct LightningChunks;
// short_conv.cu: causal convolution per channel + silu over columns p [T, C] (row pitch ld). w [taps, C], ring [slots, taps, C]: position p at p mod taps
constexpr int kMaxTaps = 8;
struct ConvArgs {
  const void* p;
  long long ld;
  int C, taps;
  const float *w, *b;  // b: [C] or nullptr
  float* ring;
  const long long* slots;
  const int *row_seq, *q_start, *q_len, *positions;
  int rows, num_seqs;
  void* out;  // [T, C]
};
int launch_short_conv(const ConvArgs& a, bool is_f32, cudaStream_t st);

// mamba.cu: Mamba-2. Projection rows p [T, ld] = z (H dv) | x (H dv) | B (G dn) | C (G dn) | dt (H), widths multiples of 8
struct MambaArgs {
  const void* p;
  long long ld;
  int H, dn, dv, G, dv_real, norm_groups, dt_at;
  const void* xbc;  // convolved and activated x | B | C [T, H dv + 2 G dn] (nullptr: the decode step convolves itself)
  int taps;
  const float *conv_w, *conv_b;
  float* ring;
  const float *dt_bias, *neg_a, *D, *norm_w;  // [H] each, norm [H dv]
  float* state;                               // [slots, H, dn, dv]
  const long long* slots;
  const int *q_start, *q_len, *positions;
  int num_seqs, rows;
  float eps;
  float* y;   // fp32 [T, H dv]
  void* out;  // [T, H dv], padding columns zeroed by the caller
  float *dt, *cum;  // chunked form: fp32 [T, H]
};
int launch_mamba2_recurrent(const MambaArgs& a, bool is_f32, cudaStream_t st);  // xbc == nullptr: one row per sequence
int launch_mamba2_chunked(const MambaArgs& a, const LightningChunks& c, int chunk, cudaStream_t st);

// delta.cu: gated delta rule. Projection rows p [T, ld]: q (G dk) | k (G dk) | v (H dv) | beta (H) at beta_at; z [T, H dk] fp32: argument of the decays without dt_bias;
// gate [T, H dv]: logits of the output gate, fp32 in the decode step, else of the rows' type
struct DeltaArgs {
  const void* p;
  long long ld;
  int H, G, dk, dv, dv_real, beta_at;
  const float* z;
  long long ld_z;
  const void* gate;
  long long ld_gate;
  const void* qkv;  // convolved and activated q | k | v [T, 2 G dk + H dv] (nullptr: the decode step convolves itself)
  int taps;
  const float* conv_w;
  float* ring;
  const float *dt_bias, *neg_a, *norm_w;  // [H dk], [H], [dv]
  float* state;                           // [slots, H, dk, dv]
  const long long* slots;
  const int *q_start, *q_len, *positions;
  int num_seqs, rows;
  float q_scale, unit_eps, eps, mult;
  float* o;  // fp32 [T, H dv]
  void* out;
  long long ld_out;
};
struct DeltaChunks {
  const int *seq, *row0, *len;  // per chunk
  const int *first, *count;     // per sequence
  int n_chunks, chunk;
  void* images;  // [n_chunks, H, delta_image_bytes]: scaled queries and keys, causal matrix, (I + M)^-1 beta, decay over the chunk
  int tiles;     // (set by the launch)
};
int launch_delta_recurrent(const DeltaArgs& a, bool is_f32, cudaStream_t st);  // qkv == nullptr: one row per sequence, norm and gate in the launch
int64_t delta_image_bytes(int dk, int chunk);
int launch_delta_chunked(const DeltaArgs& a, DeltaChunks c, cudaStream_t st);

// mixed.cu: attention with mixed scores over wide cache rows k [pages, 1, page, KV dk], v [pages, 1, page, KV dv]
struct MixedDecodeArgs {
  const void* q;  // [B, H dk]
  long long q_stride;
  const float* mix;  // [H, H] (to, from)
  const void *kc, *vc;
  const int* bt;
  int bt_stride;
  const int* ctx;
  void* out;
  float *part_o, *part_ml;  // [B, H, splits, dv], [B, H, splits, 2] (splits > 1)
  int B, H, KV, dk, dv, page;
  float scale;
  int window, splits;
  AttnExtra x;
};
bool mixed_decode_supported(int H, int KV, int dk, int dv);
int mixed_decode_ctas(int H, int KV, int dk, int dv);  // CTAs per SM
int launch_mixed_decode(const MixedDecodeArgs& a, cudaStream_t st);
void launch_decode_merge(const float* po, const float* pml, void* out, int B, int H, int dv, int splits, AttnExtra x, cudaStream_t st);  // attention.cu
// out [T, H * pitch], pitch >= KV * dk (columns behind it are the caller's)
int launch_fold_heads(const void* q, long long q_stride, const float* mix, void* out, int pitch, int T, int H, int KV, int dk, bool is_f32, cudaStream_t st);

// a2a.cu: expert-parallel all-to-all over peer memory (see the file comment for the protocol)
struct A2AParams {
  int size, rank;
  int ne;                        // experts per rank (<= 128)
  int cap;                       // rows of a receive region = most (token, slot) pairs one rank can send (its rows * k)
  unsigned long long recv[8];    // every rank's receive area: bf16 [size regions][cap][H]
  unsigned long long meta[8];    // every rank's int32 [size][2 * ne]: rows per expert and first grouped row at the sender
  unsigned long long flags[8];   // every rank's uint32 [16]: dispatch epochs [0..8), return epochs [8..16)
  unsigned long long ret[8];     // every rank's return buffer: bf16 [cap][H]
  int* status;
};
void launch_a2a_dispatch(const A2AParams* p, const void* x, const int* perm, const int* offsets, int rows, int k, int H, unsigned epoch, cudaStream_t st);
void launch_a2a_receive(const A2AParams* p, unsigned epoch, int* local_offsets, int* seg, void* xs, int max_rows, int H, cudaStream_t st);
void launch_a2a_return(const A2AParams* p, const int* local_offsets, const int* seg, const void* ys, int max_rows, int H, unsigned epoch, cudaStream_t st);
void launch_a2a_wait(const A2AParams* p, unsigned epoch, cudaStream_t st);

// latent.cu: latent attention (compressed key / value cache); see the file comment for the layouts. is_f32: every tensor is fp32
struct LatentGeom {
  int H, dk, dn, R, Rp, dr, drp;   // heads; padded q columns per head, its unrotated part; latent size, padded; rotated size, padded in the cache
  int dv, Kp;                      // value size per head, latent columns of the value weights (32-padded)
  int off_c, off_r, off_g;         // column offsets in the projection rows: latent, rotated key (-1: queries only), gate (-1: no gate)
};
struct LatentPrep {
  const int* positions;
  const long long* slots;
  const float *norm_w, *cos_t, *sin_t;
  int half, max_pos;
  void *c_cache, *r_cache;
  float eps;
};
void launch_latent_prepare(void* p, long long ld, int rows, const LatentPrep& pr, const LatentGeom& g, bool is_f32, cudaStream_t st);
void launch_latent_gather(const void* c_cache, const void* r_cache, const int* bt, int bt_stride, int page, const int* seq, const int* key0,
                          const int* n_keys, const int* row0, int num_seqs, int max_rows, void* c_out, int c_pitch, void* r_out, int r_pitch, int Rp, int drp,
                          cudaStream_t st);
void launch_latent_absorb(const void* p, long long ld, const int* row_idx, int rows, const void* wuk, void* q_lat, const LatentGeom& g,
                          const LatentPrep* prep, cudaStream_t st);
struct LatentDecodeArgs {
  const void *q_lat, *c_cache, *r_cache;
  const int* bt;
  int bt_stride;
  const int *row_seq, *row_ctx;
  int rows, page;
  float scale;
  const float* sink;       // [H] (nullptr: none)
  int window, splits;      // splits: a power of two
  void* o_lat;             // bf16 [rows, H, Rp]: result when the splits of a row are one cluster
  float *part_o, *part_ml; // else fp32 [rows, H, clusters, Rp] and [rows, H, clusters, 2]
};
int latent_cluster_size(int splits);
extern int g_latent_head_groups;
int launch_latent_decode(const LatentDecodeArgs& a, const LatentGeom& g, cudaStream_t st);
void launch_latent_expand(const LatentDecodeArgs& a, const int* row_idx, const void* wuv, const void* p, long long ld, void* out, int out_pitch,
                          const LatentGeom& g, cudaStream_t st);
int launch_latent_rows_f32(const float* p, long long ld, const int* row_idx, const int* row_seq, const int* row_ctx, int rows, const float* wuk,
                           const float* wuv, const float* c_cache, const float* r_cache, const int* bt, int bt_stride, float* out, int out_pitch,
                           const LatentGeom& g, int page, float scale, int window, const float* sink, cudaStream_t st);
void launch_linear_f32(const float* x, int ldx, const float* w, const float* bias, float* out, int ldo, int M, int N, int K, cudaStream_t st);
// w stacks experts [N, K]; items: work list of launch_moe_items with 64 rows per item
void launch_grouped_linear_f32(const float* x, int ldx, const float* w, float* out, int ldo, const int* items, int n_items, int N, int K, cudaStream_t st);

// attention_tc.cu, latent layout: q [T, H * dk] (pitch q_pitch), k [kv_rows, H * kn] and v [kv_rows, H * DV] with one pitch, kr [kv_rows, dk - kn]
struct LatentTcArgs {
  const void *q, *k, *v, *kr;
  long long T, kv_rows;
  int q_pitch, kv_pitch, kr_pitch;
  int H, dk, kn, dv;
  const int *q_start, *q_len, *ctx, *kv_row0, *tile_seq, *tile_q0;  // ctx: keys of a sequence in k / v (its query rows are the last q_len)
  int num_tiles;
  void* out;
  int out_pitch;
  const void* gate;
  int gate_pitch;
  const float* sink;
  float scale;
  int window;
  int* status;
};
int prefill_latent_tc_dv(int dk, int dv);
int prefill_latent_tc_tile_rows(int dv_padded);
int launch_prefill_latent_tc(const LatentTcArgs& a, cudaStream_t st);

// elementwise.cu, fp32 residual stream
void launch_bigram_embedding(const void* table, const void* bigram, const int* ids, const int* prev, float* out, int rows, int W, int vocab, int buckets,
                             long long mul_prev, long long mul_cur, float scale, void* out2, long long ld2, bool is_f32, cudaStream_t st);
void launch_add_layernorm(float* residual, const float* delta, const float* w1, const float* b1, void* y1, const float* w2, const float* b2, void* y2,
                          int rows, int W, int y_pitch, float eps, bool is_f32, cudaStream_t st);
void launch_sandwich_norm(float* residual, const void* sub, long long ld_sub, bool sub_f32, const int* pos, const float* wts, int k, const float* w_sub,
                          bool sub_one, float mult, const float* w_next, bool next_one, bool rms, void* y, long long ld_y, int rows, int W, int y_width, float eps,
                          bool vec, bool is_f32, cudaStream_t st);
void launch_rope_pairs_kv(void* qkv, long long ld, const int* positions, const long long* slots, const float* cos_t, const float* sin_t, void* k_cache,
                          void* v_cache, int T, int H, int KV, int dk, int dv, int page, int half, int max_pos, bool is_f32, cudaStream_t st);

// elementwise.cu: per-head norm, half rotation and cache write of projection rows p [T, ld] (columns: queries 0, keys off_k, values off_v)
struct RopeHeadsArgs {
  void* p;
  long long ld;
  int off_k, off_v;  // off_v == off_k: the values are the projected keys
  const int* positions;
  const long long* slots;
  const float *cos_t, *sin_t;  // [max_pos, half]
  void *k_cache, *v_cache;
  int T, H, KV, dk, dv, dim, page, half, max_pos;  // dim: real columns of a head (the norm's divisor)
  const float *q_norm, *k_norm;                    // [dk] or nullptr
  float eps;
  int wide;             // a cache row holds all heads of a token ([pages, 1, page, KV * width])
  const void* v_first;  // values to blend with, row pitch ld_first (nullptr: none)
  long long ld_first;
  float lam;
};
int launch_rope_heads_kv(const RopeHeadsArgs& a, bool is_f32, cudaStream_t st);

// streams.cu: several residual streams per token
constexpr int kMaxStreams = 16;
struct StreamArgs {
  float* streams;  // [T, S, W]
  int S, W;
  const int* ids;  // given: the streams start from rows of sub = the embedding table [vocab, ld_sub], normed with w_open
  int vocab;
  const float* w_open;
  const void* sub;  // output of the sublayer, rows of ld_sub (nullptr: nothing to write back)
  long long ld_sub;
  const int* pos;  // [T, k] rows of an expert-ordered sub, with weights wts [T, k]
  const float* wts;
  int k;
  const float *mix, *write;  // [S, S] (from, to), [S]
  int keep;                  // the streams are read again
  const float* read;         // [S] (nullptr: ones)
  const float* w_next;       // [W] (nullptr: no norm)
  void* y;
  long long ld_y;
  int y_width;
  float eps;
  int vec;  // rows, pitches and pointers allow four-column accesses
};
int launch_stream_step(const StreamArgs& a, int rows, bool is_f32, cudaStream_t st);

// lightning.cu: linear attention with one constant decay per head. Projection rows p [T, ld] = q (H dk) | k (H dk) | v (H dv) | g (H dv) at the given
// first columns, widths multiples of 8. The chunked form overwrites q, k and v with their activations.
struct LightningArgs {
  const void* p;
  long long ld;
  int H, dk, dv, off_k, off_v, off_g;
  const float* powers;  // [H, chunk + 2]: decay^0 .. decay^chunk, then what fp32 loses of decay^1
  int off_q, qk_div;    // first column of the queries; head h uses query / key head h / qk_div
  const float *cum, *vscale;  // launch_decayed_chunks: [rows, H] running sums of the base-2 log decays inside a chunk, weights of the values
  int chunk;
  float* state;  // [slots, H, dk, dv]
  const long long* slots;
  const int *q_start, *q_len, *positions;
  int num_seqs, rows;
  float* o;  // fp32 [T, H dv]
  // norm and gate
  const float* norm_w;  // [H dv]
  int real;             // real columns of all heads (the norm's divisor)
  float eps, mult;
  void* out;
  long long ld_out;
};
struct LightningChunks {
  const int *seq, *row0, *len;  // per chunk
  const int *first, *count;     // per sequence
  int n_chunks;
  float* added;   // [n_chunks, H, dk, dv]: what each chunk adds to the state
  void* states;   // bf16 [n_chunks, H, 2, dk, dv]: the state in front of each chunk, high and low parts
};
int launch_lightning_recurrent(const LightningArgs& a, bool is_f32, cudaStream_t st);
int launch_lightning_chunked(const LightningArgs& a, const LightningChunks& c, cudaStream_t st);
int launch_decayed_chunks(const LightningArgs& a, const LightningChunks& c, cudaStream_t st);  // outputs in a.o, no activation, norm or gate

// gla.cu: gated linear attention. Projection rows p [T, ld] = q (H dk) | k (H dk) | v (H dv) | g (H dv) | a (rank), widths multiples of 8
struct GlaArgs {
  const void* p;
  long long ld;
  int H, dk, dv, dv_real, rank, off_k, off_v, off_g, off_a;
  const float *a2, *a2_bias, *norm_w;  // [H dk, rank], [H dk], [dv]
  float* state;                        // [slots, H, dk, dv]
  const long long* slots;              // per sequence
  const int *q_start, *q_len, *positions;
  int num_seqs, rows;
  float q_scale, inv_tau, eps;
  float* o;   // fp32 [T, H dv] (unused by the fused decode step)
  void* out;  // [T, H dv]
};
struct GlaChunks {
  const int *seq, *row0, *len;    // per chunk
  const int *first, *count;       // per sequence
  int n_chunks, chunk;
  void* qk;      // bf16 [T, H, 4, dk]: scaled queries (high, low part), scaled keys (high, low part)
  void* a;       // bf16 [n_chunks, H, 2, chunk, chunk]
  float* decay;  // [n_chunks, H, dk]
};
int launch_gla_recurrent(const GlaArgs& a, bool fused, bool is_f32, cudaStream_t st);
int launch_gla_chunked(const GlaArgs& a, const GlaChunks& c, cudaStream_t st);
void launch_gated_act(const void* in, long long ld_in, void* out, long long ld_out, int rows, int I, int act, bool is_f32, cudaStream_t st);

// aux.cu
void launch_lora_delta(const void* x, int ldx, const void* A, const void* Bs, void* y, int ldy, int M, int K, int N, int r, cudaStream_t st);
void launch_pool(const void* h, int H, const int* start, const int* len, int S, int mode, int normalize, float* out, cudaStream_t st);
void launch_softmax_rows(const float* x, float* y, int rows, int C, cudaStream_t st);
void launch_tq_encode(const void* x, int src_dtype, long long rows, int dim, int pdim, int bits, const float* signs, const float* edges, uint8_t* codes,
                      float* norms, cudaStream_t st);
void launch_tq_decode(const uint8_t* codes, const float* norms, long long rows, int dim, int pdim, int bits, const float* signs, const float* centroids,
                      void* out, int dst_dtype, cudaStream_t st);
// lz4_block.cpp (host)
size_t lz4_compress_bound(size_t n);
size_t lz4_compress(const uint8_t* src, size_t n, uint8_t* dst, size_t cap);
size_t lz4_decompress(const uint8_t* src, size_t n, uint8_t* dst, size_t n_out);

// quant.cu
void launch_q4_quantize(const void* w, int src_dtype, long long n_blocks, uint8_t* packed, float* scales, cudaStream_t st);
void launch_q4_dequantize(const uint8_t* packed, const float* scales, long long n_blocks, void* out, int dst_dtype, cudaStream_t st);

}  // namespace dlv
