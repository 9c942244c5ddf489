// Linear attention with one constant decay per head ("lightning attention"): q, k, v pass through silu, then per head
//   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t;
// the heads of a row are RMS-normed together and gated with a sigmoid. State, decays, scores and outputs are fp32; the activated rows are
// of the projections' type.
//
//   lightning_recurrent_kernel  token by token, one CTA per (64 value columns, head, sequence), its part of the state in registers: decode
//                               steps, the 32-bit form of prompts, and key widths the chunked form does not take.
//   Prompts in chunks of 128 tokens. Nothing walks the chunks one by one but an elementwise kernel:
//   lightning_act_kernel        the activations, in place (every CTA of the kernels below reads rows that others read too);
//   lightning_chunk_kv_kernel   per (chunk, head, 64 value columns): what the chunk adds to the state, sum_s decay^(end - s) k_s v_s^T;
//   lightning_scan_kernel       per (sequence, head, element): the state in front of every chunk, the slot's new state;
//   lightning_chunk_out_kernel  per (chunk, head, 64 value columns): decay^(t + 1) S^T q_t plus the causal part inside the chunk, whose weights
//                               (q_t . k_s) decay^(t - s) go from the accumulators of the first product into the second.
//   What is fp32 by definition (weighted values, state, weights) enters the tensor cores as pairs of bf16 numbers (high and low part, 16 bits of
//   mantissa) with fp32 accumulation; the activated q, k, v are exact in bf16.
//   lightning_norm_gate_kernel  norm over all heads of a row, output gate.
// With decays that are data (DATA: one number per token and head, running sums of their base-2 logarithms inside the chunk in `cum`, values weighted by
// `vscale`, queries and keys shared by groups of heads) the same three kernels are the chunked form of Mamba-2 (mamba.cu), without activation and norm.
#include "common.cuh"
#include "gemm_api.h"
#include "io.cuh"
#include "mma_pair.cuh"

namespace dlv {

namespace {

constexpr int kLnCols = 64;    // value columns per CTA
constexpr int kLnChunk = 128;  // tokens per chunk

// silu; bf16 rows are activated into bf16, the type the tensor cores read (both evaluation orders see the same numbers)
__device__ __forceinline__ float ln_act(float z, const float*) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float ln_act(float z, const __nv_bfloat16*) { return bf2f(f2bf(__fdividef(z, 1.f + __expf(-z)))); }

}  // namespace

// =====================================================================================================================
// Recurrent form. 256 threads = 16 column groups (4 value columns each) x 16 row groups; thread (cx, rg) owns state rows rg, rg + 16, ..
// =====================================================================================================================
template <typename TIO, int RPT>
__global__ void __launch_bounds__(256) lightning_recurrent_kernel(const LightningArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float sq[RPT * 16], sk[RPT * 16];
  __shared__ float red[8][kLnCols];
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int cx = tid & 15, rg = tid >> 4, c0 = blockIdx.x * kLnCols + cx * 4;
  const bool col_ok = c0 < a.dv;
  const int row0 = a.q_start[s], n = a.q_len[s];
  if (n == 0) return;
  const TIO* p = static_cast<const TIO*>(a.p);
  float* state = a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * a.dk * a.dv + c0;
  const bool fresh = a.positions[row0] == 0;  // a sequence that starts at position 0 starts from a zero state
  const float* pw = a.powers + static_cast<size_t>(h) * (a.chunk + 2);
  const float al = pw[1], al_lo = pw[a.chunk + 1];  // the decay as a sum of two fp32 numbers: hundreds of steps do not drift
  float st[RPT][4];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + 16 * i;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh && col_ok && d < a.dk) v = *reinterpret_cast<const float4*>(state + static_cast<size_t>(d) * a.dv);
    st[i][0] = v.x; st[i][1] = v.y; st[i][2] = v.z; st[i][3] = v.w;
  }
  for (int t = 0; t < n; ++t) {
    const TIO* row = p + static_cast<size_t>(row0 + t) * a.ld;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (col_ok) {
      io_ld4(row + a.off_v + h * a.dv + c0, v);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = ln_act(v[e], row);
    }
    for (int d = tid; d < RPT * 16; d += 256) {
      float q = 0.f, k = 0.f;
      if (d < a.dk) {
        q = ln_act(io_ld(row + h * a.dk + d), row);
        k = ln_act(io_ld(row + a.off_k + h * a.dk + d), row);
      }
      sq[d] = q;
      sk[d] = k;
    }
    __syncthreads();
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + 16 * i;
      const float k = sk[d], q = sq[d];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        st[i][e] = fmaf(st[i][e], al, fmaf(st[i][e], al_lo, k * v[e]));
        o[e] += st[i][e] * q;
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    if ((tid & 31) < 16) *reinterpret_cast<float4*>(&red[tid >> 5][cx * 4]) = make_float4(o[0], o[1], o[2], o[3]);
    __syncthreads();  // (also: everyone is done with sq and sk)
    if (tid < kLnCols) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[w][tid];
      const int c = blockIdx.x * kLnCols + tid;
      if (c < a.dv) a.o[static_cast<size_t>(row0 + t) * (a.H * a.dv) + h * a.dv + c] = sum;
    }
  }
  if (!col_ok) return;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + 16 * i;
    if (d < a.dk) *reinterpret_cast<float4*>(state + static_cast<size_t>(d) * a.dv) = make_float4(st[i][0], st[i][1], st[i][2], st[i][3]);
  }
}

// one CTA per row: RMS norm over the heads together, plain weight, times sigmoid(gate) and a constant
template <typename TIO>
__global__ void __launch_bounds__(256) lightning_norm_gate_kernel(const LightningArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  const int t = blockIdx.x, n = a.H * a.dv;
  const float* o = a.o + static_cast<size_t>(t) * n;
  const TIO* g = static_cast<const TIO*>(a.p) + static_cast<size_t>(t) * a.ld + a.off_g;
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < n; c += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(o + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float inv = rsqrtf(block_sum(ss, red) / a.real + a.eps);
  TIO* out = static_cast<TIO*>(a.out) + static_cast<size_t>(t) * a.ld_out;
  for (int c = threadIdx.x * 4; c < n; c += blockDim.x * 4) {
    float v[4], w[4], z[4];
    io_ld4(o + c, v);
    io_ld4(a.norm_w + c, w);
    io_ld4(g + c, z);
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = v[e] * inv * w[e] * a.mult / (1.f + expf(-z[e]));
    io_st4(out + c, v);
  }
}

static int launch_norm_gate(const LightningArgs& a, bool is_f32, cudaStream_t st) {
  const int n = a.H * a.dv, threads = n >= 1024 ? 256 : (n >= 512 ? 128 : 64);
  const cudaError_t e = is_f32 ? launch_pdl(lightning_norm_gate_kernel<float>, dim3(a.rows), dim3(threads), 0, st, a)
                               : launch_pdl(lightning_norm_gate_kernel<__nv_bfloat16>, dim3(a.rows), dim3(threads), 0, st, a);
  return e == cudaSuccess ? 0 : 2;
}

template <typename TIO>
static int launch_recurrent_t(const LightningArgs& a, cudaStream_t st) {
  const dim3 grid((a.dv + kLnCols - 1) / kLnCols, a.H, a.num_seqs);
  cudaError_t e;
  if (a.dk <= 32) e = launch_pdl(lightning_recurrent_kernel<TIO, 2>, grid, dim3(256), 0, st, a);
  else if (a.dk <= 64) e = launch_pdl(lightning_recurrent_kernel<TIO, 4>, grid, dim3(256), 0, st, a);
  else if (a.dk <= 128) e = launch_pdl(lightning_recurrent_kernel<TIO, 8>, grid, dim3(256), 0, st, a);
  else if (a.dk <= 256) e = launch_pdl(lightning_recurrent_kernel<TIO, 16>, grid, dim3(256), 0, st, a);
  else e = launch_pdl(lightning_recurrent_kernel<TIO, 32>, grid, dim3(256), 0, st, a);
  return e == cudaSuccess ? 0 : 2;
}

int launch_lightning_recurrent(const LightningArgs& a, bool is_f32, cudaStream_t st) {
  if (a.rows == 0 || a.num_seqs == 0) return 0;
  if (a.dk > 512) return 1;
  const int rc = is_f32 ? launch_recurrent_t<float>(a, st) : launch_recurrent_t<__nv_bfloat16>(a, st);
  return rc != 0 ? rc : launch_norm_gate(a, is_f32, st);
}

// =====================================================================================================================
// Chunked form. NK: 16-channel tiles of the key width (padded)
// =====================================================================================================================
// q, k and v of every row are activated once, in place: columns [0, n) of the projection rows
__global__ void __launch_bounds__(256) lightning_act_kernel(const LightningArgs a, __nv_bfloat16* p, int n) {
  pdl_wait();
  pdl_trigger();
  const unsigned per = static_cast<unsigned>(n) / 8, i = blockIdx.x * 256u + threadIdx.x;
  if (i >= per * static_cast<unsigned>(a.rows)) return;
  __nv_bfloat16* at = p + static_cast<size_t>(i / per) * a.ld + (i % per) * 8;
  float v[8];
  io_ld8(at, v);
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = ln_act(v[e], at);
  io_st8(at, v);
}

// copy of a [kLnChunk][16 NK] tile of rows, started here; columns behind dk and rows behind len become zero
template <int NK>
__device__ __forceinline__ void copy_tile(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int len, int dk) {
  constexpr int P = NK * 16 + 8, CH = NK * 2;
  for (int e = threadIdx.x; e < kLnChunk * CH; e += 256) {
    const int t = e / CH, x = (e % CH) * 8;
    const bool ok = t < len && x < dk;
    cp16(smem_u32(dst + t * P + x), src + (ok ? t * ld + x : 0), ok);
  }
}

constexpr int kLnPV = kLnCols + 8;  // row pitch of value and state tiles

template <int NK>
struct LnKv {
  static constexpr int P = NK * 16 + 8;
  static constexpr int kBytes = (kLnChunk * P + 2 * kLnChunk * kLnPV) * 2 + (2 * kLnChunk + 4) * 4;
};
template <int NK>
struct LnOut {
  static constexpr int P = NK * 16 + 8;
  static constexpr int kBytes = (kLnChunk * P + kLnChunk * kLnPV + 2 * NK * 16 * kLnPV) * 2 + (2 * kLnChunk + 4) * 4;
  static_assert(kBytes <= 227 * 1024, "tiles must fit shared memory");
};

__device__ __forceinline__ float ln_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// DATA: the chunk's running sums and value weights (zero behind its end: a weight of one that meets zero rows)
__device__ __forceinline__ void load_decays(const LightningArgs& a, int row0, int len, int h, float* cum, float* vs) {
  for (int i = threadIdx.x; i < kLnChunk; i += 256) {
    const size_t at = static_cast<size_t>(row0 + (i < len ? i : 0)) * a.H + h;
    cum[i] = i < len ? a.cum[at] : 0.f;
    vs[i] = i < len ? a.vscale[at] : 0.f;
  }
}

template <int NK, bool DATA>
__global__ void __launch_bounds__(256) lightning_chunk_kv_kernel(const LightningArgs a, const LightningChunks c) {
  pdl_wait();
  pdl_trigger();
  using L = LnKv<NK>;
  extern __shared__ __align__(16) uint8_t lsm[];
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(lsm);      // [128][P]
  __nv_bfloat16* sV = sK + kLnChunk * L::P;                       // [2][128][kLnPV] decay^(len - 1 - t) v_t, high and low parts
  float* pw = reinterpret_cast<float*>(sV + 2 * kLnChunk * kLnPV);  // decay^0 ..; DATA: running sums, then value weights
  const int ck = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kLnCols, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row0 = c.row0[ck], len = c.len[ck], dk = a.dk, dv = a.dv;
  const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(a.p) + static_cast<size_t>(row0) * a.ld;
  if constexpr (DATA) load_decays(a, row0, len, h, pw, pw + kLnChunk);
  else
    for (int i = tid; i <= kLnChunk; i += 256) pw[i] = a.powers[static_cast<size_t>(h) * (kLnChunk + 2) + i];
  copy_tile<NK>(sK, p + a.off_k + h / a.qk_div * dk, a.ld, len, dk);
  cp_commit();
  __syncthreads();
  for (int e = tid; e < kLnChunk * 8; e += 256) {
    const int t = e >> 3, x = (e & 7) * 8;
    uint32_t hi[4] = {0u, 0u, 0u, 0u}, lo[4] = {0u, 0u, 0u, 0u};
    if (t < len && c0 + x < dv) {
      const uint4 u = *reinterpret_cast<const uint4*>(p + t * a.ld + a.off_v + h * dv + c0 + x);
      const uint32_t w[4] = {u.x, u.y, u.z, u.w};
      const float s = DATA ? ln_ex2(pw[len - 1] - pw[t]) * pw[kLnChunk + t] : pw[len - 1 - t];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = unpack_bf162(w[i]);
        split2(f.x * s, f.y * s, hi[i], lo[i]);
      }
    }
    *reinterpret_cast<uint4*>(sV + t * kLnPV + x) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(sV + (kLnChunk + t) * kLnPV + x) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  cp_wait<0>();
  __syncthreads();
  // rows = key channels (16 per tile), columns = value columns: a warp takes MT row tiles x NT column tiles of 8
  constexpr int WM = NK < 8 ? NK : 8, WN = 8 / WM, MT = NK / WM, NT = 8 / WN;
  const int wm = warp % WM, wn = warp / WM, g = lane >> 2, t4 = lane & 3;
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
  const uint32_t k_at = smem_u32(sK + ((lane & 7) + (lane >> 4) * 8) * L::P + wm * MT * 16 + ((lane >> 3) & 1) * 8);
  const uint32_t v_at = smem_u32(sV + ((lane & 7) + ((lane >> 3) & 1) * 8) * kLnPV + wn * NT * 8 + (lane >> 4) * 8);
  const int steps = (len + 15) / 16;
  for (int ks = 0; ks < steps; ++ks) {
    uint32_t kf[MT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) ldm_x4_t(k_at + (ks * 16 * L::P + m * 16) * 2, kf[m]);
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t bh[4], bl[4];
      ldm_x4_t(v_at + (ks * 16 * kLnPV + np * 16) * 2, bh);
      ldm_x4_t(v_at + ((kLnChunk + ks * 16) * kLnPV + np * 16) * 2, bl);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        mma16816(acc[m][2 * np], kf[m], bh[0], bh[1]);
        mma16816(acc[m][2 * np + 1], kf[m], bh[2], bh[3]);
        mma16816(acc[m][2 * np], kf[m], bl[0], bl[1]);
        mma16816(acc[m][2 * np + 1], kf[m], bl[2], bl[3]);
      }
    }
  }
  float* u = c.added + (static_cast<size_t>(ck) * a.H + h) * dk * dv;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int d = (wm * MT + m) * 16 + g, col = c0 + (wn * NT + n) * 8 + 2 * t4;
      if (col >= dv) continue;
      if (d < dk) *reinterpret_cast<float2*>(u + static_cast<size_t>(d) * dv + col) = make_float2(acc[m][n][0], acc[m][n][1]);
      if (d + 8 < dk) *reinterpret_cast<float2*>(u + static_cast<size_t>(d + 8) * dv + col) = make_float2(acc[m][n][2], acc[m][n][3]);
    }
}

// a thread keeps four elements of a state and walks the sequence's chunks, four loads ahead; the state in front of every chunk is left as
// two bf16 planes (high and low parts), the operands of the next kernel
template <bool DATA>
__global__ void __launch_bounds__(256) lightning_scan_kernel(const LightningArgs a, const LightningChunks c) {
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.y, s = blockIdx.z, n = c.count[s], first = c.first[s];
  const size_t per = static_cast<size_t>(a.dk) * a.dv, at = (static_cast<size_t>(blockIdx.x) * 256 + threadIdx.x) * 4;
  if (n == 0 || at >= per) return;
  float4* slot = reinterpret_cast<float4*>(a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * per + at);
  float4 st = make_float4(0.f, 0.f, 0.f, 0.f);
  if (a.positions[a.q_start[s]] != 0) st = *slot;
  const float* pw = DATA ? nullptr : a.powers + static_cast<size_t>(h) * (kLnChunk + 2);
  auto chunk = [&](int i) { return reinterpret_cast<const float4*>(c.added + (static_cast<size_t>(first + i) * a.H + h) * per + at); };
  __nv_bfloat16* planes = static_cast<__nv_bfloat16*>(c.states);
  constexpr int AHEAD = 4;
  float4 u[AHEAD];
#pragma unroll
  for (int j = 0; j < AHEAD; ++j) u[j] = j < n ? *chunk(j) : st;
  for (int i0 = 0; i0 < n; i0 += AHEAD) {
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int i = i0 + j;
      if (i >= n) break;
      const float4 add = u[j];
      if (i + AHEAD < n) u[j] = *chunk(i + AHEAD);
      uint32_t h0, h1, l0, l1;
      split2(st.x, st.y, h0, l0);
      split2(st.z, st.w, h1, l1);
      __nv_bfloat16* hi = planes + (static_cast<size_t>(first + i) * a.H + h) * 2 * per + at;
      *reinterpret_cast<uint2*>(hi) = make_uint2(h0, h1);
      *reinterpret_cast<uint2*>(hi + per) = make_uint2(l0, l1);
      const int len = c.len[first + i];
      const float d = DATA ? ln_ex2(a.cum[static_cast<size_t>(c.row0[first + i] + len - 1) * a.H + h]) : pw[len];
      st = make_float4(fmaf(st.x, d, add.x), fmaf(st.y, d, add.y), fmaf(st.z, d, add.z), fmaf(st.w, d, add.w));
    }
  }
  *slot = st;
}

template <int NK, bool DATA>
__global__ void __launch_bounds__(256, (NK <= 8 ? 2 : 1)) lightning_chunk_out_kernel(const LightningArgs a, const LightningChunks c) {
  pdl_wait();
  pdl_trigger();
  using L = LnOut<NK>;
  constexpr int P = L::P;
  extern __shared__ __align__(16) uint8_t lsm[];
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(lsm);  // [128][P]
  __nv_bfloat16* sV = sK + kLnChunk * P;                      // [128][kLnPV]
  __nv_bfloat16* sS = sV + kLnChunk * kLnPV;                  // [2][16 NK][kLnPV] state in front of the chunk, high and low parts
  float* pw = reinterpret_cast<float*>(sS + 2 * NK * 16 * kLnPV);
  const int ck = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kLnCols, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row0 = c.row0[ck], len = c.len[ck], dk = a.dk, dv = a.dv;
  const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(a.p) + static_cast<size_t>(row0) * a.ld;
  const __nv_bfloat16* state = static_cast<const __nv_bfloat16*>(c.states) + (static_cast<size_t>(ck) * a.H + h) * 2 * dk * dv;
  for (int e = tid; e < 2 * NK * 16 * 8; e += 256) {
    const int d = (e >> 3) % (NK * 16), x = (e & 7) * 8, plane = e / (NK * 16 * 8);
    const bool ok = d < dk && c0 + x < dv;
    cp16(smem_u32(sS + (plane * NK * 16 + d) * kLnPV + x), state + (ok ? (static_cast<size_t>(plane) * dk + d) * dv + c0 + x : 0), ok);
  }
  cp_commit();
  copy_tile<NK>(sK, p + a.off_k + h / a.qk_div * dk, a.ld, len, dk);
  for (int e = tid; e < kLnChunk * 8; e += 256) {
    const int t = e >> 3, x = (e & 7) * 8;
    const bool ok = t < len && c0 + x < dv;
    cp16(smem_u32(sV + t * kLnPV + x), p + (ok ? t * a.ld + a.off_v + h * dv + c0 + x : 0), ok);
  }
  cp_commit();
  if constexpr (DATA) load_decays(a, row0, len, h, pw, pw + kLnChunk);
  else
    for (int i = tid; i <= kLnChunk; i += 256) pw[i] = a.powers[static_cast<size_t>(h) * (kLnChunk + 2) + i];
  const int r0 = warp * 16, g = lane >> 2, t4 = lane & 3;  // this warp's token rows
  const bool mine = r0 < len;
  uint32_t q[NK][4];  // query fragments, straight from the rows
  {
    const bool ok0 = r0 + g < len, ok1 = r0 + g + 8 < len;
    const __nv_bfloat16* qa = p + a.off_q + h / a.qk_div * dk + static_cast<long long>(ok0 ? r0 + g : 0) * a.ld + 2 * t4;
    const __nv_bfloat16* qb = p + a.off_q + h / a.qk_div * dk + static_cast<long long>(ok1 ? r0 + g + 8 : 0) * a.ld + 2 * t4;
#pragma unroll
    for (int kt = 0; kt < NK; ++kt) {
      const bool lo = kt * 16 < dk, hi = kt * 16 + 8 < dk;  // (widths are multiples of 8)
      q[kt][0] = ok0 && lo ? *reinterpret_cast<const uint32_t*>(qa + kt * 16) : 0u;
      q[kt][1] = ok1 && lo ? *reinterpret_cast<const uint32_t*>(qb + kt * 16) : 0u;
      q[kt][2] = ok0 && hi ? *reinterpret_cast<const uint32_t*>(qa + kt * 16 + 8) : 0u;
      q[kt][3] = ok1 && hi ? *reinterpret_cast<const uint32_t*>(qb + kt * 16 + 8) : 0u;
    }
  }
  cp_wait<1>();
  __syncthreads();
  float o[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  // ---- what the state contributes: decay^(t + 1) q_t S
  if (mine) {
    const uint32_t s_at = smem_u32(sS + ((lane & 7) + ((lane >> 3) & 1) * 8) * kLnPV + (lane >> 4) * 8);
#pragma unroll
    for (int kt = 0; kt < NK; ++kt)
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t bh[4], bl[4];
        ldm_x4_t(s_at + (kt * 16 * kLnPV + np * 16) * 2, bh);
        ldm_x4_t(s_at + ((NK * 16 + kt * 16) * kLnPV + np * 16) * 2, bl);
        mma16816(o[2 * np], q[kt], bh[0], bh[1]);
        mma16816(o[2 * np + 1], q[kt], bh[2], bh[3]);
        mma16816(o[2 * np], q[kt], bl[0], bl[1]);
        mma16816(o[2 * np + 1], q[kt], bl[2], bl[3]);
      }
  }
  cp_wait<0>();
  __syncthreads();
  if (!mine) return;
  const float b0 = DATA ? pw[r0 + g] : 0.f, b1 = DATA ? pw[r0 + g + 8] : 0.f;
  const float d0 = DATA ? ln_ex2(b0) : pw[r0 + g + 1], d1 = DATA ? ln_ex2(b1) : pw[min(r0 + g + 9, kLnChunk)];
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    o[n][0] *= d0;
    o[n][1] *= d0;
    o[n][2] *= d1;
    o[n][3] *= d1;
  }
  // ---- inside the chunk: 16 keys at a time, up to the diagonal
  const uint32_t k_at = smem_u32(sK + ((lane & 7) + (lane >> 4) * 8) * P + ((lane >> 3) & 1) * 8);
  const uint32_t v_at = smem_u32(sV + ((lane & 7) + ((lane >> 3) & 1) * 8) * kLnPV + (lane >> 4) * 8);
  for (int j = 0; j <= warp; ++j) {
    float sc[2][4] = {};
#pragma unroll
    for (int kt = 0; kt < NK; ++kt) {
      uint32_t k[4];
      ldm_x4(k_at + (j * 16 * P + kt * 16) * 2, k);
      mma16816(sc[0], q[kt], k[0], k[1]);
      mma16816(sc[1], q[kt], k[2], k[3]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = j * 16 + n * 8 + 2 * t4 + (e & 1), back = r0 + g + (e >> 1) * 8 - key;
        if constexpr (DATA) sc[n][e] = back >= 0 ? sc[n][e] * ln_ex2(((e >> 1) ? b1 : b0) - pw[key]) * pw[kLnChunk + key] : 0.f;
        else sc[n][e] = back >= 0 ? sc[n][e] * pw[back] : 0.f;
      }
    uint32_t ph[4], pl[4];
    split2(sc[0][0], sc[0][1], ph[0], pl[0]);
    split2(sc[0][2], sc[0][3], ph[1], pl[1]);
    split2(sc[1][0], sc[1][1], ph[2], pl[2]);
    split2(sc[1][2], sc[1][3], ph[3], pl[3]);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      uint32_t b[4];
      ldm_x4_t(v_at + (j * 16 * kLnPV + np * 16) * 2, b);
      mma16816(o[2 * np], ph, b[0], b[1]);
      mma16816(o[2 * np + 1], ph, b[2], b[3]);
      mma16816(o[2 * np], pl, b[0], b[1]);
      mma16816(o[2 * np + 1], pl, b[2], b[3]);
    }
  }
  float* out = a.o + static_cast<size_t>(row0) * (a.H * dv) + h * dv + c0;
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    const int col = n * 8 + 2 * t4;
    if (c0 + col >= dv) continue;
    if (r0 + g < len) *reinterpret_cast<float2*>(out + static_cast<size_t>(r0 + g) * (a.H * dv) + col) = make_float2(o[n][0], o[n][1]);
    if (r0 + g + 8 < len) *reinterpret_cast<float2*>(out + static_cast<size_t>(r0 + g + 8) * (a.H * dv) + col) = make_float2(o[n][2], o[n][3]);
  }
}

template <int NK, bool DATA>
static cudaError_t launch_chunked_t(const LightningArgs& a, const LightningChunks& c, cudaStream_t st) {
  static PerDeviceOnce once;
  cudaError_t e = cudaSuccess;
  if (once.first()) {
    e = cudaFuncSetAttribute(lightning_chunk_kv_kernel<NK, DATA>, cudaFuncAttributeMaxDynamicSharedMemorySize, LnKv<NK>::kBytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(lightning_chunk_out_kernel<NK, DATA>, cudaFuncAttributeMaxDynamicSharedMemorySize, LnOut<NK>::kBytes);
    if (e != cudaSuccess) return e;
  }
  if constexpr (!DATA) {
    const int n = a.off_v + a.H * a.dv;
    const unsigned vecs = static_cast<unsigned>(n) / 8 * static_cast<unsigned>(a.rows);
    e = launch_pdl(lightning_act_kernel, dim3((vecs + 255) / 256), dim3(256), 0, st, a, static_cast<__nv_bfloat16*>(const_cast<void*>(a.p)), n);
    if (e != cudaSuccess) return e;
  }
  const dim3 grid(c.n_chunks, a.H, (a.dv + kLnCols - 1) / kLnCols);
  e = launch_pdl(lightning_chunk_kv_kernel<NK, DATA>, grid, dim3(256), LnKv<NK>::kBytes, st, a, c);
  if (e != cudaSuccess) return e;
  const unsigned blocks = static_cast<unsigned>((static_cast<size_t>(a.dk) * a.dv / 4 + 255) / 256);
  e = launch_pdl(lightning_scan_kernel<DATA>, dim3(blocks, a.H, a.num_seqs), dim3(256), 0, st, a, c);
  if (e != cudaSuccess) return e;
  return launch_pdl(lightning_chunk_out_kernel<NK, DATA>, grid, dim3(256), LnOut<NK>::kBytes, st, a, c);
}

template <bool DATA>
static cudaError_t launch_chunked(const LightningArgs& a, const LightningChunks& c, cudaStream_t st) {
  if (a.dk <= 32) return launch_chunked_t<2, DATA>(a, c, st);
  if (a.dk <= 64) return launch_chunked_t<4, DATA>(a, c, st);
  if (a.dk <= 128) return launch_chunked_t<8, DATA>(a, c, st);
  return launch_chunked_t<16, DATA>(a, c, st);
}

int launch_lightning_chunked(const LightningArgs& a, const LightningChunks& c, cudaStream_t st) {
  if (a.rows == 0 || c.n_chunks == 0) return 0;
  if (a.off_k != a.H * a.dk || a.off_v != 2 * a.off_k || static_cast<long long>(a.rows) * (a.off_v + a.H * a.dv) / 8 > 0xffffff00ll) return 1;
  if (a.dk > 256 || a.chunk != kLnChunk || (a.dv + kLnCols - 1) / kLnCols > 65535) return 1;
  return launch_chunked<false>(a, c, st) != cudaSuccess ? 2 : launch_norm_gate(a, false, st);
}

int launch_decayed_chunks(const LightningArgs& a, const LightningChunks& c, cudaStream_t st) {
  if (a.rows == 0 || c.n_chunks == 0) return 0;
  if (a.dk > 256 || a.chunk != kLnChunk || a.cum == nullptr || a.vscale == nullptr || a.qk_div < 1) return 1;
  return launch_chunked<true>(a, c, st) != cudaSuccess ? 2 : 0;
}

}  // namespace dlv
