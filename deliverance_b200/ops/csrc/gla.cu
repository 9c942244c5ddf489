// Gated linear attention: per head  S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t  with a decay per key channel,
// log a = log(sigmoid(z)) / tau, z = W_a2 (low-rank input) + bias; the heads are RMS-normed over the value columns and gated with silu(g).
// State, decays and everything that enters the recurrence besides the projections are fp32 (chunked form: pairs of bf16 numbers, high and
// low part, multiplied on the tensor cores with fp32 accumulation; 16 bits of mantissa).
//
//   gla_recurrent_kernel  one CTA per (64 value columns, head, sequence): the CTA's part of the state stays in registers while it walks the
//                         sequence's rows of this batch. Decode steps (one row) also norm and gate: the CTAs of a head form a cluster and
//                         exchange their sums of squares through distributed shared memory. Also the 32-bit form of prompts.
//   gla_prepare_kernel    prompts, all (chunk, head) pairs at once: decays and their running sums b inside the chunk, q exp(b),
//                         k exp(b_end - b), the chunk's causal matrix A[t, s] = sum_d q_t k_s exp(b_t - b_s). A is one product of
//                         q exp(b) and k exp(-b) unless a channel's decay over the chunk would leave the fp32 range (then term by term).
//   gla_chunks_kernel     one CTA per (64 value columns, head, sequence) walks the chunks: O^T = S^T Q^T + V^T A^T, then
//                         S^T = S^T diag(exp(b_end)) + V^T K. S^T is the accumulator of the second product and, converted in registers,
//                         the left operand of the first; eight warps = 4 x 16 value columns x 2 halves of the key channels, whose shares
//                         of O meet in shared memory; chunk tiles arrive by cp.async in two stages.
//   gla_norm_gate_kernel  norm and gate of prompt rows.
#include <cooperative_groups.h>

#include "common.cuh"
#include "gemm_api.h"
#include "mma_pair.cuh"

namespace dlv {

namespace {

__device__ __forceinline__ float g_ld(const float* p) { return *p; }
__device__ __forceinline__ float g_ld(const __nv_bfloat16* p) { return bf2f(*p); }
__device__ __forceinline__ void g_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void g_st(__nv_bfloat16* p, float v) { *p = f2bf(v); }
__device__ __forceinline__ float4 g_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 g_ld4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf162(u.x), b = unpack_bf162(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void g_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void g_st4(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf162(v.x, v.y), pack_bf162(v.z, v.w)); }

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }

constexpr int kGlaCols = 64;  // value columns per CTA

}  // namespace

// =====================================================================================================================
// Recurrent form. 256 threads = 16 column groups (4 value columns each) x 16 row groups; thread (cx, rg) owns state rows rg, rg + 16, ..
// =====================================================================================================================
template <typename TIO, int RPT, bool FUSED>
__global__ void __launch_bounds__(256) gla_recurrent_kernel(const GlaArgs a) {
  pdl_wait();
  pdl_trigger();
  namespace cg = cooperative_groups;
  __shared__ float sq[RPT * 16], sk[RPT * 16], sa[RPT * 16];
  __shared__ float red[8][kGlaCols];
  __shared__ float sx[1024];  // low-rank decay input of the row
  __shared__ float ssum, half_sum;  // sum of squares of this CTA's columns, of its upper half
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int cx = tid & 15, rg = tid >> 4, c0 = blockIdx.x * kGlaCols + cx * 4;
  const bool col_ok = c0 < a.dv;
  const int row0 = a.q_start[s], n = a.q_len[s];
  if (n == 0 && !FUSED) return;
  const TIO* p = static_cast<const TIO*>(a.p);
  float* state = a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * a.dk * a.dv + c0;
  const bool fresh = a.positions[row0] == 0;  // a sequence that starts at position 0 starts from a zero state
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
    for (int r = tid; r < a.rank; r += 256) sx[r] = g_ld(row + a.off_a + r);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col_ok) v = g_ld4(row + a.off_v + h * a.dv + c0);
    __syncthreads();
    for (int d = tid; d < RPT * 16; d += 256) {
      float q = 0.f, k = 0.f, al = 0.f;
      if (d < a.dk) {
        q = g_ld(row + h * a.dk + d) * a.q_scale;
        k = g_ld(row + a.off_k + h * a.dk + d);
        const float* w = a.a2 + static_cast<size_t>(h * a.dk + d) * a.rank;
        float z = a.a2_bias[h * a.dk + d];
        for (int r = 0; r < a.rank; r += 4) {
          const float4 wv = *reinterpret_cast<const float4*>(w + r);
          z += wv.x * sx[r] + wv.y * sx[r + 1] + wv.z * sx[r + 2] + wv.w * sx[r + 3];
        }
        al = expf(log_sigmoid(z) * a.inv_tau);
      }
      sq[d] = q;
      sk[d] = k;
      sa[d] = al;
    }
    __syncthreads();
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + 16 * i;
      const float al = sa[d], k = sk[d], q = sq[d];
      st[i][0] = st[i][0] * al + k * v.x;
      st[i][1] = st[i][1] * al + k * v.y;
      st[i][2] = st[i][2] * al + k * v.z;
      st[i][3] = st[i][3] * al + k * v.w;
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] += st[i][e] * q;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    if ((tid & 31) < 16) *reinterpret_cast<float4*>(&red[tid >> 5][cx * 4]) = make_float4(o[0], o[1], o[2], o[3]);
    __syncthreads();
    if (tid < kGlaCols) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[w][tid];
      const int c = blockIdx.x * kGlaCols + tid;
      if constexpr (FUSED) {
        red[0][tid] = sum;
        float ss = warp_sum(sum * sum);
        if (tid == 32) half_sum = ss;
        asm volatile("bar.sync 1, 64;" ::: "memory");
        if (tid == 0) ssum = ss + half_sum;
      } else if (c < a.dv) {
        a.o[static_cast<size_t>(row0 + t) * (a.H * a.dv) + h * a.dv + c] = sum;
      }
    }
  }
  if (col_ok && n > 0) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + 16 * i;
      if (d < a.dk) *reinterpret_cast<float4*>(state + static_cast<size_t>(d) * a.dv) = make_float4(st[i][0], st[i][1], st[i][2], st[i][3]);
    }
  }
  if constexpr (FUSED) {
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    float ss = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) ss += *cluster.map_shared_rank(&ssum, r);
    const int c = blockIdx.x * kGlaCols + tid;
    if (tid < kGlaCols && c < a.dv && n > 0) {
      const float inv = rsqrtf(ss / a.dv_real + a.eps);
      const float g = g_ld(p + static_cast<size_t>(row0) * a.ld + a.off_g + h * a.dv + c);
      g_st(static_cast<TIO*>(a.out) + static_cast<size_t>(row0) * (a.H * a.dv) + h * a.dv + c, red[0][tid] * inv * a.norm_w[c] * silu(g));
    }
    cluster.sync();  // no CTA leaves while another one may still read its sum
  }
}

// one warp per (row, head)
template <typename TIO>
__global__ void __launch_bounds__(256) gla_norm_gate_kernel(const GlaArgs a) {
  pdl_wait();
  pdl_trigger();
  const long long w = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(a.rows) * a.H) return;
  const int t = static_cast<int>(w / a.H), h = static_cast<int>(w % a.H);
  const size_t base = static_cast<size_t>(t) * (a.H * a.dv) + h * a.dv;
  const float* o = a.o + base;
  const TIO* g = static_cast<const TIO*>(a.p) + static_cast<size_t>(t) * a.ld + a.off_g + h * a.dv;
  float ss = 0.f;
  for (int c = lane * 4; c < a.dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(o + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float inv = rsqrtf(warp_sum(ss) / a.dv_real + a.eps);
  TIO* out = static_cast<TIO*>(a.out) + base;
  for (int c = lane * 4; c < a.dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(o + c), nw = *reinterpret_cast<const float4*>(a.norm_w + c), gv = g_ld4(g + c);
    g_st4(out + c, make_float4(v.x * inv * nw.x * silu(gv.x), v.y * inv * nw.y * silu(gv.y), v.z * inv * nw.z * silu(gv.z), v.w * inv * nw.w * silu(gv.w)));
  }
}

template <typename TIO, bool FUSED>
static int launch_recurrent_t(const GlaArgs& a, cudaStream_t st) {
  const int slices = (a.dv + kGlaCols - 1) / kGlaCols;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, a.H, a.num_seqs);
  cfg.blockDim = dim3(256);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = g_pdl_enabled ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = FUSED ? slices : 1;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  cudaError_t e;
  if (a.dk <= 32) e = cudaLaunchKernelEx(&cfg, gla_recurrent_kernel<TIO, 2, FUSED>, a);
  else if (a.dk <= 64) e = cudaLaunchKernelEx(&cfg, gla_recurrent_kernel<TIO, 4, FUSED>, a);
  else if (a.dk <= 128) e = cudaLaunchKernelEx(&cfg, gla_recurrent_kernel<TIO, 8, FUSED>, a);
  else if (a.dk <= 256) e = cudaLaunchKernelEx(&cfg, gla_recurrent_kernel<TIO, 16, FUSED>, a);
  else e = cudaLaunchKernelEx(&cfg, gla_recurrent_kernel<TIO, 32, FUSED>, a);
  return e == cudaSuccess ? 0 : 2;
}

int launch_gla_recurrent(const GlaArgs& a, bool fused, bool is_f32, cudaStream_t st) {
  if (a.rows == 0 || a.num_seqs == 0) return 0;
  if (a.dk > 512 || a.rank > 1024 || (fused && a.dv > 8 * kGlaCols)) return 1;
  if (fused) return is_f32 ? launch_recurrent_t<float, true>(a, st) : launch_recurrent_t<__nv_bfloat16, true>(a, st);
  const int rc = is_f32 ? launch_recurrent_t<float, false>(a, st) : launch_recurrent_t<__nv_bfloat16, false>(a, st);
  if (rc != 0) return rc;
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(a.rows) * a.H + 7) / 8));
  if (is_f32) launch_pdl(gla_norm_gate_kernel<float>, grid, dim3(256), 0, st, a);
  else launch_pdl(gla_norm_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a);
  return 0;
}

// =====================================================================================================================
// Chunked form
// =====================================================================================================================
// The chunked form keeps decay logarithms in base 2 (their sums are the arguments of the special-function unit, without a further rounding).
constexpr float kGlaMaxLogDecay = 86.f;  // 2^(+-86) and its products with projections stay inside fp32
__device__ __forceinline__ float exp2_sfu(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// log2(sigmoid(z)) = min(z, 0) log2(e) - log2(1 + e^-|z|); log(1 + x) = 2 artanh(x / (2 + x)) by the series of the inverse hyperbolic tangent,
// whose argument is at most 1 / 3 here (eight terms: a relative error of 1e-8)
__device__ __forceinline__ float log2_sigmoid(float z) {
  constexpr float log2e = 1.4426950408889634f;
  const float x = exp2_sfu(-fabsf(z) * log2e), s = __fdividef(x, 2.f + x), s2 = s * s;
  float p = fmaf(s2, 1.f / 15.f, 1.f / 13.f);
  p = fmaf(s2, p, 1.f / 11.f);
  p = fmaf(s2, p, 1.f / 9.f);
  p = fmaf(s2, p, 1.f / 7.f);
  p = fmaf(s2, p, 1.f / 5.f);
  p = fmaf(s2, p, 1.f / 3.f);
  p = fmaf(s2, p, 1.f);
  return (fminf(z, 0.f) - 2.f * s * p) * log2e;
}

template <int C>
__global__ void __launch_bounds__(256) gla_prepare_kernel(const GlaArgs a, const GlaChunks c) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t gsm[];
  const int ck = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dk = a.dk, dk16 = (dk + 15) / 16 * 16, P = dk16 + 8;
  float* sb = reinterpret_cast<float*>(gsm);                               // [C][dk] decay logarithms, then their running sums
  float* sx = sb + C * dk;                                                 // [C][16] part of the low-rank decay input
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sx + C * 16);       // [2][C][P] q exp(b), high and low parts
  __nv_bfloat16* sK = sQ + 2 * C * P;                                      // [2][C][P] k exp(-b)
  const int row0 = c.row0[ck], len = c.len[ck];
  const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(a.p);
  // ---- decay logarithms: a thread keeps one channel and takes every ng-th token
  const int ng = 256 / dk, d_own = tid % dk, grp = tid / dk;
  for (int r0 = 0; r0 < a.rank; r0 += 16) {
    const int nr = min(16, a.rank - r0);  // 8 or 16 columns of the decay input per round
    __syncthreads();
    for (int e = tid; e < C * 4; e += 256) {
      const int t = e >> 2, x = (e & 3) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (t < len && x < nr) v = g_ld4(p + static_cast<size_t>(row0 + t) * a.ld + a.off_a + r0 + x);
      *reinterpret_cast<float4*>(sx + t * 16 + x) = v;
    }
    __syncthreads();
    if (grp < ng) {
      const float* wp = a.a2 + static_cast<size_t>(h * dk + d_own) * a.rank + r0;
      float4 w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) w[i] = i * 4 < nr ? *reinterpret_cast<const float4*>(wp + i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float bias = r0 == 0 ? a.a2_bias[h * dk + d_own] : 0.f;
      const bool last = r0 + 16 >= a.rank;
#pragma unroll 4
      for (int t = grp; t < C; t += ng) {
        float z = r0 == 0 ? bias : sb[t * dk + d_own];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 x = *reinterpret_cast<const float4*>(sx + t * 16 + i * 4);
          z += (w[i].x * x.x + w[i].y * x.y) + (w[i].z * x.z + w[i].w * x.w);
        }
        if (last) z = t < len ? log2_sigmoid(z) * a.inv_tau : 0.f;
        sb[t * dk + d_own] = z;
      }
    }
  }
  __syncthreads();
  for (int d = tid; d < dk; d += 256) {
    float acc = 0.f;
#pragma unroll 8
    for (int t = 0; t < C; ++t) {
      acc += sb[t * dk + d];
      sb[t * dk + d] = acc;
    }
  }
  __syncthreads();
  const float* b_end = sb + (C - 1) * dk;
  bool small = true;
  for (int d = tid; d < dk; d += 256) small = small && b_end[d] > -kGlaMaxLogDecay;
  const bool fast = __syncthreads_and(small);
  // ---- scaled queries and keys
  __nv_bfloat16* qk = static_cast<__nv_bfloat16*>(c.qk);
  const int half = dk / 2, ng2 = 256 / half, grp2 = tid / half, d2 = (tid % half) * 2;  // a thread keeps one pair of channels
  if (grp2 < ng2) {
    const float2 be = *reinterpret_cast<const float2*>(b_end + d2);
    const __nv_bfloat16* col = p + static_cast<size_t>(row0) * a.ld + h * dk + d2;
    uint32_t* dst = reinterpret_cast<uint32_t*>(qk + (static_cast<size_t>(row0) * a.H + h) * 4 * dk + d2);
    const size_t step = static_cast<size_t>(a.H) * 2 * dk;  // (in pairs)
#pragma unroll 4
    for (int t = grp2; t < C; t += ng2) {
      uint32_t qu = 0u, ku = 0u;
      if (t < len) {
        qu = *reinterpret_cast<const uint32_t*>(col + t * a.ld);
        ku = *reinterpret_cast<const uint32_t*>(col + t * a.ld + a.off_k);
      }
      const float2 q = unpack_bf162(qu), k = unpack_bf162(ku), b = *reinterpret_cast<const float2*>(sb + t * dk + d2);
      uint32_t qh, ql, kh, kl;
      split2(q.x * a.q_scale * exp2_sfu(b.x), q.y * a.q_scale * exp2_sfu(b.y), qh, ql);
      split2(k.x * exp2_sfu(be.x - b.x), k.y * exp2_sfu(be.y - b.y), kh, kl);
      if (t < len) {
        uint32_t* row = dst + t * step;
        row[0] = qh;
        row[half] = ql;
        row[2 * half] = kh;
        row[3 * half] = kl;
      }
      if (fast) {
        *reinterpret_cast<uint32_t*>(sQ + t * P + d2) = qh;
        *reinterpret_cast<uint32_t*>(sQ + (C + t) * P + d2) = ql;
        split2(k.x * exp2_sfu(-b.x), k.y * exp2_sfu(-b.y), kh, kl);
        *reinterpret_cast<uint32_t*>(sK + t * P + d2) = kh;
        *reinterpret_cast<uint32_t*>(sK + (C + t) * P + d2) = kl;
      }
    }
  }
  if (dk16 != dk)
    for (int e = tid; e < 2 * C * 4; e += 256) {
      reinterpret_cast<uint32_t*>(sQ + (e >> 2) * P + dk)[e & 3] = 0u;
      reinterpret_cast<uint32_t*>(sK + (e >> 2) * P + dk)[e & 3] = 0u;
    }
  for (int d = tid; d < dk; d += 256) c.decay[(static_cast<size_t>(ck) * a.H + h) * dk + d] = exp2_sfu(b_end[d]);
  __syncthreads();
  // ---- causal matrix of the chunk: the 16 x 16 blocks on and below the diagonal
  __nv_bfloat16* am = static_cast<__nv_bfloat16*>(c.a) + (static_cast<size_t>(ck) * a.H + h) * 2 * C * C;
  if (fast) {
    constexpr int NB = C / 16;
    const int g = lane >> 2, t4 = lane & 3;
    for (int blk = warp; blk < NB * NB; blk += 8) {
      const int mb = blk / NB, nb = blk % NB;
      if (nb > mb) continue;
      float acc[2][4] = {};
      const uint32_t q_at = smem_u32(sQ + (mb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * P + (lane >> 4) * 8);
      const uint32_t k_at = smem_u32(sK + (nb * 16 + (lane & 7) + (lane >> 4) * 8) * P + ((lane >> 3) & 1) * 8);
      const uint32_t lo = static_cast<uint32_t>(C * P * 2);
      for (int k16 = 0; k16 < dk16 / 16; ++k16) {
        uint32_t qh[4], ql[4], kh[4], kl[4];
        ldm_x4(q_at + k16 * 32, qh);
        ldm_x4(q_at + lo + k16 * 32, ql);
        ldm_x4(k_at + k16 * 32, kh);
        ldm_x4(k_at + lo + k16 * 32, kl);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma16816(acc[n], qh, kh[2 * n], kh[2 * n + 1]);
          mma16816(acc[n], qh, kl[2 * n], kl[2 * n + 1]);
          mma16816(acc[n], ql, kh[2 * n], kh[2 * n + 1]);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = mb * 16 + g + 8 * r, s = nb * 16 + n * 8 + 2 * t4;
          uint32_t hi, lw;
          split2(s <= t ? acc[n][2 * r] : 0.f, s + 1 <= t ? acc[n][2 * r + 1] : 0.f, hi, lw);
          *reinterpret_cast<uint32_t*>(am + t * C + s) = hi;
          *reinterpret_cast<uint32_t*>(am + C * C + t * C + s) = lw;
        }
    }
  } else {
    for (int e = tid; e < C * C / 2; e += 256) {
      const int t = e / (C / 2), s = (e % (C / 2)) * 2;
      if (s / 16 > t / 16) continue;
      float v[2] = {0.f, 0.f};
      if (t < len) {
        const __nv_bfloat16* q = p + static_cast<size_t>(row0 + t) * a.ld + h * dk;
        for (int j = 0; j < 2; ++j) {
          if (s + j > t) continue;
          const __nv_bfloat16* k = p + static_cast<size_t>(row0 + s + j) * a.ld + a.off_k + h * dk;
          float acc = 0.f;
          for (int d = 0; d < dk; ++d) acc += bf2f(q[d]) * bf2f(k[d]) * exp2_sfu(sb[t * dk + d] - sb[(s + j) * dk + d]);
          v[j] = acc * a.q_scale;
        }
      }
      uint32_t hi, lw;
      split2(v[0], v[1], hi, lw);
      *reinterpret_cast<uint32_t*>(am + t * C + s) = hi;
      *reinterpret_cast<uint32_t*>(am + C * C + t * C + s) = lw;
    }
  }
}

// NK: 16-channel tiles of the key width (padded). Stage layout in shared memory: q high | q low | k high | k low [C][P], v [C][72],
// A high | low [C][C + 8], decay [16 NK] fp32.
template <int C, int NK>
struct GlaStage {
  static constexpr int P = NK * 16 + 8, PV = kGlaCols + 8, PA = C + 8;
  static constexpr int kV = 4 * C * P * 2;
  static constexpr int kA = kV + C * PV * 2;
  static constexpr int kDec = kA + 2 * C * PA * 2;
  static constexpr int kBytes = (kDec + NK * 16 * 4 + 127) / 128 * 128;
  static constexpr int PO = kGlaCols + 4;
  static constexpr int kTotal = 2 * kBytes + 2 * C * PO * 4;  // two stages, both halves' shares of the outputs
  static_assert(NK % 2 == 0 && kTotal <= 227 * 1024, "two stages must fit shared memory");
};

template <int C, int NK>
__global__ void __launch_bounds__(256, 1) gla_chunks_kernel(const GlaArgs a, const GlaChunks c) {
  pdl_wait();
  pdl_trigger();
  using L = GlaStage<C, NK>;
  constexpr int NH = NK / 2;  // 16-channel tiles per warp
  extern __shared__ __align__(128) uint8_t gsm[];
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t4 = lane & 3, wd = warp & 3, hk = warp >> 2;  // 16 value columns, half of the key channels
  float* so = reinterpret_cast<float*>(gsm + 2 * L::kBytes);
  const int c0 = blockIdx.x * kGlaCols, n_chunks = c.count[s], first = c.first[s];
  if (n_chunks == 0) return;
  const int dk = a.dk, dv = a.dv;
  const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(a.p);
  const __nv_bfloat16* qk = static_cast<const __nv_bfloat16*>(c.qk);
  const __nv_bfloat16* am = static_cast<const __nv_bfloat16*>(c.a);
  float* state = a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * dk * dv;
  const bool fresh = a.positions[a.q_start[s]] == 0;

  auto load = [&](int i, int stage) {
    const int ck = first + i, row0 = c.row0[ck], len = c.len[ck];
    const uint32_t base = smem_u32(gsm + stage * L::kBytes);
    constexpr int CH = NK * 2;  // 16-byte chunks per row and plane
    for (int e = tid; e < 4 * C * CH; e += 256) {
      const int x = e % CH, t = (e / CH) % C, plane = e / (CH * C);
      const bool ok = t < len && x * 8 < dk;
      const __nv_bfloat16* src = qk + ((static_cast<size_t>(row0 + (ok ? t : 0)) * a.H + h) * 4 + plane) * dk + (ok ? x * 8 : 0);
      cp16(base + ((plane * C + t) * L::P + x * 8) * 2, src, ok);
    }
    for (int e = tid; e < C * 8; e += 256) {
      const int t = e >> 3, x = (e & 7) * 8;
      const bool ok = t < len && c0 + x < dv;
      cp16(base + L::kV + (t * L::PV + x) * 2, p + static_cast<size_t>(row0 + (ok ? t : 0)) * a.ld + a.off_v + h * dv + (ok ? c0 + x : 0), ok);
    }
    const __nv_bfloat16* ap = am + (static_cast<size_t>(ck) * a.H + h) * 2 * C * C;
    for (int e = tid; e < 2 * C * (C / 8); e += 256) {
      const int r = e / (C / 8), x = (e % (C / 8)) * 8;
      cp16(base + L::kA + (r * L::PA + x) * 2, ap + r * C + x, true);
    }
    for (int e = tid; e < NK * 4; e += 256) cp16(base + L::kDec + e * 16, c.decay + (static_cast<size_t>(ck) * a.H + h) * dk + (e * 4 < dk ? e * 4 : 0), e * 4 < dk);
    cp_commit();
  };

  load(0, 0);
  // S^T: rows = value columns (16 per warp), columns = key channels
  float st[2 * NH][4];
  const int vr = c0 + wd * 16 + g, d_at = hk * NH * 16 + 2 * t4;
#pragma unroll
  for (int j = 0; j < 2 * NH; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d_at + j * 8 + (e & 1), col = vr + (e >> 1) * 8;
      st[j][e] = (!fresh && d < dk && col < dv) ? state[static_cast<size_t>(d) * dv + col] : 0.f;
    }
  for (int i = 0; i < n_chunks; ++i) {
    if (i + 1 < n_chunks) {
      load(i + 1, (i + 1) & 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const uint32_t base = smem_u32(gsm + (i & 1) * L::kBytes);
    const float* dec = reinterpret_cast<const float*>(gsm + (i & 1) * L::kBytes + L::kDec);
    float o[C / 8][4];
#pragma unroll
    for (int j = 0; j < C / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    // O^T = S^T Q^T
    const uint32_t q_at = base + (((lane & 7) + (lane >> 4) * 8) * L::P + hk * NH * 16 + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int kt = 0; kt < NH; ++kt) {
      uint32_t sh[4], sl[4];
      split2(st[2 * kt][0], st[2 * kt][1], sh[0], sl[0]);
      split2(st[2 * kt][2], st[2 * kt][3], sh[1], sl[1]);
      split2(st[2 * kt + 1][0], st[2 * kt + 1][1], sh[2], sl[2]);
      split2(st[2 * kt + 1][2], st[2 * kt + 1][3], sh[3], sl[3]);
#pragma unroll
      for (int np = 0; np < C / 16; ++np) {
        uint32_t b[4];
        ldm_x4(q_at + (np * 16 * L::P + kt * 16) * 2, b);
        mma16816(o[2 * np], sh, b[0], b[1]);
        mma16816(o[2 * np + 1], sh, b[2], b[3]);
        mma16816(o[2 * np], sl, b[0], b[1]);
        mma16816(o[2 * np + 1], sl, b[2], b[3]);
        ldm_x4(q_at + ((C + np * 16) * L::P + kt * 16) * 2, b);
        mma16816(o[2 * np], sh, b[0], b[1]);
        mma16816(o[2 * np + 1], sh, b[2], b[3]);
      }
    }
    // O^T += V^T A^T (the halves take every other block of tokens)
    uint32_t vf[C / 16][4];
#pragma unroll
    for (int ks = 0; ks < C / 16; ++ks) {
      ldm_x4_t(base + L::kV + ((ks * 16 + (lane & 7) + (lane >> 4) * 8) * L::PV + wd * 16 + ((lane >> 3) & 1) * 8) * 2, vf[ks]);
      if ((ks & 1) != hk) continue;
#pragma unroll
      for (int np = ks; np < C / 16; ++np) {
        const uint32_t at = base + L::kA + ((np * 16 + (lane & 7) + (lane >> 4) * 8) * L::PA + ks * 16 + ((lane >> 3) & 1) * 8) * 2;
        uint32_t b[4];
        ldm_x4(at, b);
        mma16816(o[2 * np], vf[ks], b[0], b[1]);
        mma16816(o[2 * np + 1], vf[ks], b[2], b[3]);
        ldm_x4(at + C * L::PA * 2, b);
        mma16816(o[2 * np], vf[ks], b[0], b[1]);
        mma16816(o[2 * np + 1], vf[ks], b[2], b[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < C / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) so[(hk * C + j * 8 + 2 * t4 + (e & 1)) * L::PO + wd * 16 + g + (e >> 1) * 8] = o[j][e];
    // S^T = S^T diag(decay) + V^T K
#pragma unroll
    for (int j = 0; j < 2 * NH; ++j) {
      const float2 e = *reinterpret_cast<const float2*>(dec + d_at + j * 8);
      st[j][0] *= e.x;
      st[j][1] *= e.y;
      st[j][2] *= e.x;
      st[j][3] *= e.y;
    }
    const uint32_t k_at = base + ((2 * C + (lane & 7) + ((lane >> 3) & 1) * 8) * L::P + hk * NH * 16 + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int ks = 0; ks < C / 16; ++ks)
#pragma unroll
      for (int jp = 0; jp < NH; ++jp) {
        uint32_t b[4];
        ldm_x4_t(k_at + (ks * 16 * L::P + jp * 16) * 2, b);
        mma16816(st[2 * jp], vf[ks], b[0], b[1]);
        mma16816(st[2 * jp + 1], vf[ks], b[2], b[3]);
        ldm_x4_t(k_at + ((C + ks * 16) * L::P + jp * 16) * 2, b);
        mma16816(st[2 * jp], vf[ks], b[0], b[1]);
        mma16816(st[2 * jp + 1], vf[ks], b[2], b[3]);
      }
    __syncthreads();  // the stage is refilled by the next iteration's load; both shares of the outputs are complete
    const int row0 = c.row0[first + i], len = c.len[first + i];
    for (int e = tid; e < C * (kGlaCols / 4); e += 256) {
      const int t = e / (kGlaCols / 4), x = (e % (kGlaCols / 4)) * 4;
      if (t >= len || c0 + x >= dv) continue;
      const float4 u = *reinterpret_cast<const float4*>(so + t * L::PO + x), w = *reinterpret_cast<const float4*>(so + (C + t) * L::PO + x);
      *reinterpret_cast<float4*>(a.o + static_cast<size_t>(row0 + t) * (a.H * dv) + h * dv + c0 + x) = make_float4(u.x + w.x, u.y + w.y, u.z + w.z, u.w + w.w);
    }
  }
#pragma unroll
  for (int j = 0; j < 2 * NH; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d_at + j * 8 + (e & 1), col = vr + (e >> 1) * 8;
      if (d < dk && col < dv) state[static_cast<size_t>(d) * dv + col] = st[j][e];
    }
}

template <int C, int NK>
static cudaError_t launch_chunks_t(const GlaArgs& a, const GlaChunks& c, cudaStream_t st) {
  using L = GlaStage<C, NK>;
  static PerDeviceOnce once;
  if (once.first()) {
    const cudaError_t e = cudaFuncSetAttribute(gla_chunks_kernel<C, NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kTotal);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(gla_chunks_kernel<C, NK>, dim3((a.dv + kGlaCols - 1) / kGlaCols, a.H, a.num_seqs), dim3(256), L::kTotal, st, a, c);
}

template <int C>
static cudaError_t launch_prepare_t(const GlaArgs& a, const GlaChunks& c, cudaStream_t st) {
  const int P = (a.dk + 15) / 16 * 16 + 8;
  const size_t smem = static_cast<size_t>(C * a.dk + C * 16) * 4 + static_cast<size_t>(4) * C * P * 2;
  static PerDeviceOnce once;
  if (once.first()) {
    const cudaError_t e = cudaFuncSetAttribute(gla_prepare_kernel<C>, cudaFuncAttributeMaxDynamicSharedMemorySize, 120 * 1024);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(gla_prepare_kernel<C>, dim3(c.n_chunks, a.H), dim3(256), smem, st, a, c);
}

int launch_gla_chunked(const GlaArgs& a, const GlaChunks& c, cudaStream_t st) {
  if (a.rows == 0 || c.n_chunks == 0) return 0;
  cudaError_t e;
  if (c.chunk == 64 && a.dk <= 128) e = launch_prepare_t<64>(a, c, st);
  else if (c.chunk == 32 && a.dk <= 256) e = launch_prepare_t<32>(a, c, st);
  else return 1;
  if (e == cudaSuccess) {
    if (c.chunk == 64 && a.dk <= 32) e = launch_chunks_t<64, 2>(a, c, st);
    else if (c.chunk == 64 && a.dk <= 64) e = launch_chunks_t<64, 4>(a, c, st);
    else if (c.chunk == 64) e = launch_chunks_t<64, 8>(a, c, st);
    else e = launch_chunks_t<32, 16>(a, c, st);
  }
  if (e != cudaSuccess) return 2;
  launch_pdl(gla_norm_gate_kernel<__nv_bfloat16>, dim3(static_cast<unsigned>((static_cast<long long>(a.rows) * a.H + 7) / 8)), dim3(256), 0, st, a);
  return 0;
}

}  // namespace dlv
