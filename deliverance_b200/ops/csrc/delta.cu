// Gated delta rule: per head  S <- diag(a_t) S,  u_t = beta_t (v_t - S^T k_t),  S <- S + k_t u_t^T,  o_t = S^T q_t  with a decay per key channel,
// log a = neg_a softplus(low-rank projection + dt_bias); q, k and v come through a short convolution (short_conv.cu), q and k are unit vectors (q times
// q_scale). The heads are RMS-normed over the value columns and gated with a sigmoid. State, decays, unit vectors, beta, norm and gate are fp32 (chunked
// form: pairs of bf16 numbers, high and low part, multiplied on the tensor cores with fp32 accumulation; 16 bits of mantissa).
//
//   delta_recurrent_kernel  one CTA per (64 value columns, head, sequence), its part of the state in registers. Decode steps (STEP: one row per sequence)
//                           convolve their token (the ring of inputs is updated in place), norm and gate in the same launch: the CTAs of a head form a
//                           cluster and exchange their sums of squares. Also the 32-bit form of prompts.
//   delta_prepare_kernel    prompts, all (chunk, head) pairs at once. With running sums b of the log decays inside the chunk: q exp(b), k exp(b_end - b),
//                           k exp(b), the causal matrix A[t, s] = sum_d q_t k_s exp(b_t - b_s), M[t, s] = beta_t sum_d k_t k_s exp(b_t - b_s) for s < t, and
//                           T = (I + M)^-1 diag(beta). A and M are products of q exp(b), k exp(b) with k exp(-b) unless a channel's decay over the chunk
//                           would leave the fp32 range (then term by term).
//   delta_chunks_kernel     one CTA per (64 value columns, head, sequence) walks the chunks: U^T = (V^T - S^T K'^T) T^T, O^T = S^T Q^T + U^T A^T, then
//                           S^T = S^T diag(exp(b_end)) + U^T K. S^T is the accumulator of the last product and, converted in registers, the left operand of
//                           the first two; eight warps = 4 x 16 value columns x 2 halves of the key channels. The halves' shares of S^T K'^T meet in
//                           shared memory (both then hold the whole U^T), those of O on their way out. Two stages; the prepare kernel writes what
//                           a chunk needs as it lies in shared memory, so a stage is one contiguous copy.
//   delta_norm_gate_kernel  norm and gate of prompt rows.
#include <cooperative_groups.h>

#include "common.cuh"
#include "conv_step.cuh"
#include "gemm_api.h"
#include "io.cuh"
#include "mma_pair.cuh"

namespace dlv {

namespace {

constexpr int kDnCols = 64;  // value columns per CTA
__device__ __forceinline__ float dn_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
// softplus of prepared chunks: the series of log(1 + e) where 1 + e would round e away
__device__ __forceinline__ float dn_softplus_fast(float v) {
  const float e = __expf(-fabsf(v));
  return fmaxf(v, 0.f) + (e < 0.04f ? e * (1.f - e * (0.5f - e * (0.33333333f - e * (0.25f - e * 0.2f)))) : __logf(1.f + e));
}
__device__ __forceinline__ float dn_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float dn_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

}  // namespace

// =====================================================================================================================
// Recurrent form. 256 threads = 16 column groups (4 value columns each) x 16 row groups; thread (cx, rg) owns state rows rg, rg + 16, ..
// =====================================================================================================================
template <typename TIO, int RPT, bool STEP>
__global__ void __launch_bounds__(256) delta_recurrent_kernel(const DeltaArgs a) {
  pdl_wait();
  pdl_trigger();
  namespace cg = cooperative_groups;
  __shared__ float sq[RPT * 16], sk[RPT * 16], sa[RPT * 16], sv[kDnCols], su[kDnCols];
  __shared__ float red[8][kDnCols], redq[32], redk[32];
  __shared__ float ssum, half_sum;  // sum of squares of this CTA's columns, of its upper half
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int cx = tid & 15, rg = tid >> 4, c_first = blockIdx.x * kDnCols, c0 = c_first + cx * 4;
  const bool col_ok = c0 < a.dv;
  const int row0 = a.q_start[s], n = a.q_len[s];
  if (n == 0 && !STEP) return;
  const int per_group = a.H / a.G, g = h / per_group;
  const int off_k = a.G * a.dk, off_v = 2 * off_k, C = off_v + a.H * a.dv;
  const TIO* p = static_cast<const TIO*>(a.p);
  float* state = a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * a.dk * a.dv + c0;
  const int pos0 = a.positions[row0];
  const bool fresh = pos0 == 0;  // a sequence that starts at position 0 starts from a zero state
  const float neg_a = a.neg_a[h];
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
    const float* z = a.z + static_cast<size_t>(row0 + t) * a.ld_z + h * a.dk;
    float qq = 0.f, kk = 0.f;
    if constexpr (STEP) {
      // (ring rows of a query / key head are written by its first CTA, those of value columns by their own)
      float* ring = a.ring + static_cast<size_t>(a.slots[s]) * a.taps * C;
      float* own = ring + static_cast<size_t>(pos0 % a.taps) * C;
      const bool writes = blockIdx.x == 0 && h % per_group == 0;
      for (int e = tid; e < 2 * RPT * 16 + kDnCols; e += 256) {
        if (e < 2 * RPT * 16) {
          const int d = e % (RPT * 16), c = (e < RPT * 16 ? 0 : off_k) + g * a.dk + d;
          float y = 0.f;
          if (d < a.dk) {
            const float x = io_ld(row + c);
            y = conv_step<TIO>(x, a.conv_w, nullptr, ring, a.taps, C, c, pos0);
            if (writes) own[c] = x;
          }
          (e < RPT * 16 ? sq : sk)[d] = y;
          if (e < RPT * 16) qq += y * y;
          else kk += y * y;
        } else {
          const int col = e - 2 * RPT * 16, c = off_v + h * a.dv + c_first + col;
          float y = 0.f;
          if (c_first + col < a.dv) {
            const float x = io_ld(row + c);
            y = conv_step<TIO>(x, a.conv_w, nullptr, ring, a.taps, C, c, pos0);
            own[c] = x;
          }
          sv[col] = y;
        }
      }
    } else {
      const TIO* in = static_cast<const TIO*>(a.qkv) + static_cast<size_t>(row0 + t) * C;
      for (int d = tid; d < RPT * 16; d += 256) {
        const float q = d < a.dk ? io_ld(in + g * a.dk + d) : 0.f, k = d < a.dk ? io_ld(in + off_k + g * a.dk + d) : 0.f;
        sq[d] = q;
        sk[d] = k;
        qq += q * q;
        kk += k * k;
      }
      if (tid < kDnCols) sv[tid] = c_first + tid < a.dv ? io_ld(in + off_v + h * a.dv + c_first + tid) : 0.f;
    }
    for (int d = tid; d < RPT * 16; d += 256) sa[d] = d < a.dk ? expf(neg_a * dn_softplus(z[d] + a.dt_bias[h * a.dk + d])) : 0.f;
    const float fq = rsqrtf(block_sum(qq, redq) + a.unit_eps) * a.q_scale, fk = rsqrtf(block_sum(kk, redk) + a.unit_eps);
    // ---- decay, what the state returns for the key
    float r[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + 16 * i;
      const float al = sa[d], k = sk[d];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        st[i][e] *= al;
        r[e] += st[i][e] * k;
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) r[e] += __shfl_xor_sync(0xffffffffu, r[e], 16);
    if ((tid & 31) < 16) *reinterpret_cast<float4*>(&red[tid >> 5][cx * 4]) = make_float4(r[0], r[1], r[2], r[3]);
    __syncthreads();
    if (tid < kDnCols) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[w][tid];
      su[tid] = dn_sigmoid(io_ld(row + a.beta_at + h)) * (sv[tid] - fk * sum);
    }
    __syncthreads();
    // ---- write, read
    float u[4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 4; ++e) u[e] = su[cx * 4 + e] * fk;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + 16 * i;
      const float k = sk[d], q = sq[d];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        st[i][e] += k * u[e];
        o[e] += st[i][e] * q;
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    if ((tid & 31) < 16) *reinterpret_cast<float4*>(&red[tid >> 5][cx * 4]) = make_float4(o[0], o[1], o[2], o[3]);
    __syncthreads();  // (also: everyone is done with sq, sk and sa)
    if (tid < kDnCols) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[w][tid];
      sum *= fq;
      const int c = c_first + tid;
      if constexpr (STEP) {
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
  if constexpr (STEP) {
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    float ss = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) ss += *cluster.map_shared_rank(&ssum, r);
    const int c = c_first + tid;
    if (tid < kDnCols && c < a.dv && n > 0) {
      const float inv = rsqrtf(ss / a.dv_real + a.eps) * a.mult;
      const float z = static_cast<const float*>(a.gate)[static_cast<size_t>(row0) * a.ld_gate + h * a.dv + c];
      io_st(static_cast<TIO*>(a.out) + static_cast<size_t>(row0) * a.ld_out + h * a.dv + c, red[0][tid] * inv * a.norm_w[c] * dn_sigmoid(z));
    }
    cluster.sync();  // no CTA leaves while another one may still read its sum
  }
}

// one warp per (row, head)
template <typename TIO>
__global__ void __launch_bounds__(256) delta_norm_gate_kernel(const DeltaArgs a) {
  pdl_wait();
  pdl_trigger();
  const unsigned w = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<unsigned>(a.rows) * a.H) return;
  const int t = static_cast<int>(w / a.H), h = static_cast<int>(w % a.H);
  const float* o = a.o + static_cast<size_t>(t) * (a.H * a.dv) + h * a.dv;
  const TIO* z = static_cast<const TIO*>(a.gate) + static_cast<size_t>(t) * a.ld_gate + h * a.dv;
  float ss = 0.f;
  for (int c = lane * 4; c < a.dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(o + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float inv = rsqrtf(warp_sum(ss) / a.dv_real + a.eps) * a.mult;
  TIO* out = static_cast<TIO*>(a.out) + static_cast<size_t>(t) * a.ld_out + h * a.dv;
  for (int c = lane * 4; c < a.dv; c += 128) {
    float v[4], nw[4], zv[4];
    io_ld4(o + c, v);
    io_ld4(a.norm_w + c, nw);
    io_ld4(z + c, zv);
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] *= inv * nw[e] * (sizeof(TIO) == 2 ? __fdividef(1.f, 1.f + __expf(-zv[e])) : dn_sigmoid(zv[e]));
    io_st4(out + c, v);
  }
}

static cudaError_t launch_norm_gate(const DeltaArgs& a, bool is_f32, cudaStream_t st) {
  if (static_cast<long long>(a.rows) * a.H > (1ll << 31)) return cudaErrorInvalidValue;
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(a.rows) * a.H + 7) / 8));
  return is_f32 ? launch_pdl(delta_norm_gate_kernel<float>, grid, dim3(256), 0, st, a) : launch_pdl(delta_norm_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a);
}

template <typename TIO, bool STEP>
static cudaError_t launch_recurrent_t(const DeltaArgs& a, cudaStream_t st) {
  const int slices = (a.dv + kDnCols - 1) / kDnCols;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, a.H, a.num_seqs);
  cfg.blockDim = dim3(256);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = g_pdl_enabled ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = STEP ? slices : 1;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  if (a.dk <= 32) return cudaLaunchKernelEx(&cfg, delta_recurrent_kernel<TIO, 2, STEP>, a);
  if (a.dk <= 64) return cudaLaunchKernelEx(&cfg, delta_recurrent_kernel<TIO, 4, STEP>, a);
  if (a.dk <= 128) return cudaLaunchKernelEx(&cfg, delta_recurrent_kernel<TIO, 8, STEP>, a);
  if (a.dk <= 256) return cudaLaunchKernelEx(&cfg, delta_recurrent_kernel<TIO, 16, STEP>, a);
  return cudaLaunchKernelEx(&cfg, delta_recurrent_kernel<TIO, 32, STEP>, a);
}

int launch_delta_recurrent(const DeltaArgs& a, bool is_f32, cudaStream_t st) {
  if (a.rows == 0 || a.num_seqs == 0) return 0;
  const bool step = a.qkv == nullptr;
  if (a.dk > 512 || (step && (a.dv > 8 * kDnCols || a.rows != a.num_seqs || a.taps < 1))) return 1;
  cudaError_t e;
  if (is_f32) e = step ? launch_recurrent_t<float, true>(a, st) : launch_recurrent_t<float, false>(a, st);
  else e = step ? launch_recurrent_t<__nv_bfloat16, true>(a, st) : launch_recurrent_t<__nv_bfloat16, false>(a, st);
  if (e == cudaSuccess && !step) e = launch_norm_gate(a, is_f32, st);
  return e == cudaSuccess ? 0 : 2;
}

// =====================================================================================================================
// Chunked form (decay logarithms in base 2)
// =====================================================================================================================
// What the walk reads of one (chunk, head), as it lies in shared memory: q exp(b), k exp(b_end - b), k exp(b) high | low [6][C][P], A and T high | low
// [4][C][PA], decay [16 NK] fp32. NK: 16-channel tiles of the key width (2, 4, 8 or 16); columns and rows behind the real ones are zero.
template <int C>
struct DeltaImage {
  int P, off_a, off_dec, bytes;
  static constexpr int PA = C + 8;
  __host__ __device__ constexpr explicit DeltaImage(int nk) : P(nk * 16 + 8), off_a(6 * C * (nk * 16 + 8) * 2), off_dec(0), bytes(0) {
    off_dec = off_a + 4 * C * PA * 2;
    bytes = off_dec + nk * 16 * 4;
  }
};
static int delta_tiles(int dk) { return dk <= 32 ? 2 : dk <= 64 ? 4 : dk <= 128 ? 8 : 16; }

int64_t delta_image_bytes(int dk, int chunk) { return chunk == 16 ? DeltaImage<16>(delta_tiles(dk)).bytes : DeltaImage<32>(delta_tiles(dk)).bytes; }

constexpr float kDnMaxLogDecay = 86.f;  // 2^(+-86) and its products with unit vectors stay inside fp32

template <int C, int R>
struct DeltaPrepareSmem {
  int P, off_m, off_t, off_f, bytes;
  __host__ __device__ explicit DeltaPrepareSmem(int dk) {
    P = (dk + 15) / 16 * 16 + 8;
    off_m = 6 * C * P * 2;               // [3][2][C][P]: q exp(b), k exp(-b), k exp(b); term by term: running sums [C][dk]
    off_t = off_m + 2 * C * (C + 1) * 4; // [C][C + 1] M, then its inverse
    off_f = off_t + C / R * dk * 4;      // [C / R][dk] sums of the log decays of R rows
    bytes = off_f + 3 * C * 4;           // [3][C] unit factors of q and k, beta
  }
};

// A thread keeps two channels of R rows.
template <int C, int R>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const DeltaArgs a, const DeltaChunks c) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t dsm[];
  const DeltaPrepareSmem<C, R> L(a.dk);
  constexpr int NG = C / R;
  const DeltaImage<C> I(c.tiles);
  uint8_t* image = static_cast<uint8_t*>(c.images) + (static_cast<size_t>(blockIdx.x) * a.H + blockIdx.y) * I.bytes;
  const int ck = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dk = a.dk, dk16 = (dk + 15) / 16 * 16, P = L.P, half = dk / 2;
  float* sb = reinterpret_cast<float*>(dsm);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(dsm);
  __nv_bfloat16* sK = sQ + 2 * C * P;
  __nv_bfloat16* sB = sK + 2 * C * P;
  float* sM = reinterpret_cast<float*>(dsm + L.off_m);
  float* sX = sM + C * (C + 1);
  float* sT = reinterpret_cast<float*>(dsm + L.off_t);
  float* fq = reinterpret_cast<float*>(dsm + L.off_f);
  float* fk = fq + C;
  float* beta = fk + C;
  const int row0 = c.row0[ck], len = c.len[ck], g = h / (a.H / a.G), width = 2 * a.G * dk + a.H * a.dv;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.qkv) + static_cast<size_t>(row0) * width + g * dk;
  const __nv_bfloat16* kp = qp + a.G * dk;
  const float la = a.neg_a[h] * 1.4426950408889634f;
  const int d = (tid % half) * 2, grp = tid / half, t0 = grp * R;
  const bool active = grp < NG;
  // ---- decay logarithms and their running sums inside the thread's rows
  float2 b[R];
  uint32_t qu[R], ku[R];
  if (active) {
    const float2 bias = *reinterpret_cast<const float2*>(a.dt_bias + h * dk + d);
    const float* zp = a.z + static_cast<size_t>(row0 + t0) * a.ld_z + h * dk + d;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const bool ok = t0 + i < len;
      b[i] = ok ? *reinterpret_cast<const float2*>(zp + i * a.ld_z) : make_float2(0.f, 0.f);
      qu[i] = ok ? *reinterpret_cast<const uint32_t*>(qp + static_cast<size_t>(t0 + i) * width + d) : 0u;
      ku[i] = ok ? *reinterpret_cast<const uint32_t*>(kp + static_cast<size_t>(t0 + i) * width + d) : 0u;
    }
    float2 acc = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      if (t0 + i < len) {
        acc.x += la * dn_softplus_fast(b[i].x + bias.x);
        acc.y += la * dn_softplus_fast(b[i].y + bias.y);
      }
      b[i] = acc;
    }
    *reinterpret_cast<float2*>(sT + grp * dk + d) = acc;
  }
  // ---- unit factors, one warp per row
#pragma unroll
  for (int i = 0; i < C / 8; ++i) {
    const int t = warp + 8 * i;
    float qq = 0.f, kk = 0.f;
    if (t < len)
      for (int x = lane * 4; x < dk; x += 128) {
        float q[4], k[4];
        io_ld4(qp + static_cast<size_t>(t) * width + x, q);
        io_ld4(kp + static_cast<size_t>(t) * width + x, k);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          qq += q[e] * q[e];
          kk += k[e] * k[e];
        }
      }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    if (lane == 0) {
      fq[t] = rsqrtf(qq + a.unit_eps) * a.q_scale;
      fk[t] = rsqrtf(kk + a.unit_eps);
      beta[t] = t < len ? dn_sigmoid(bf2f(static_cast<const __nv_bfloat16*>(a.p)[static_cast<size_t>(row0 + t) * a.ld + a.beta_at + h])) : 0.f;
    }
  }
  __syncthreads();
  float2 be = make_float2(0.f, 0.f);
  bool small = true;
  if (active) {
    float2 before = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const float2 v = *reinterpret_cast<const float2*>(sT + i * dk + d);
      if (i < grp) {
        before.x += v.x;
        before.y += v.y;
      }
      be.x += v.x;
      be.y += v.y;
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      b[i].x += before.x;
      b[i].y += before.y;
    }
    small = fminf(be.x, be.y) > -kDnMaxLogDecay;
    if (grp == 0) *reinterpret_cast<float2*>(image + I.off_dec + d * 4) = make_float2(dn_ex2(be.x), dn_ex2(be.y));
  }
  const bool fast = __syncthreads_and(small);
  // ---- scaled queries and keys
  if (active) {
    uint32_t* o = reinterpret_cast<uint32_t*>(image) + (t0 * I.P + d) / 2;
    const int plane = C * I.P / 2;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int t = t0 + i;
      const float2 q = unpack_bf162(qu[i]), k0 = unpack_bf162(ku[i]);
      const float uq = fq[t], uk = fk[t];
      const float2 k = make_float2(k0.x * uk, k0.y * uk);
      const float ex = dn_ex2(b[i].x), ey = dn_ex2(b[i].y);
      uint32_t qh, ql, bh, bl, kh, kl;
      split2(q.x * uq * ex, q.y * uq * ey, qh, ql);
      split2(k.x * ex, k.y * ey, bh, bl);
      split2(k.x * dn_ex2(be.x - b[i].x), k.y * dn_ex2(be.y - b[i].y), kh, kl);
      o[0] = qh;
      o[plane] = ql;
      o[2 * plane] = kh;
      o[3 * plane] = kl;
      o[4 * plane] = bh;
      o[5 * plane] = bl;
      o += I.P / 2;
      if (fast) {
        *reinterpret_cast<uint32_t*>(sQ + t * P + d) = qh;
        *reinterpret_cast<uint32_t*>(sQ + (C + t) * P + d) = ql;
        *reinterpret_cast<uint32_t*>(sB + t * P + d) = bh;
        *reinterpret_cast<uint32_t*>(sB + (C + t) * P + d) = bl;
        split2(k.x * dn_ex2(-b[i].x), k.y * dn_ex2(-b[i].y), kh, kl);
        *reinterpret_cast<uint32_t*>(sK + t * P + d) = kh;
        *reinterpret_cast<uint32_t*>(sK + (C + t) * P + d) = kl;
      } else {
        *reinterpret_cast<float2*>(sb + t * dk + d) = b[i];
      }
    }
  }
  if (const int pad = (I.P - 8 - dk) / 8; pad > 0) {
    for (int e = tid; e < 6 * C * pad; e += 256) *reinterpret_cast<uint4*>(image + ((e / pad) * I.P + dk + (e % pad) * 8) * 2) = make_uint4(0, 0, 0, 0);
    if (tid < pad * 8) reinterpret_cast<float*>(image + I.off_dec)[dk + tid] = 0.f;
  }
  if (fast && dk16 != dk)  // (widths are multiples of 8)
    for (int e = tid; e < 6 * C * 4; e += 256) reinterpret_cast<uint32_t*>(sQ + (e >> 2) * P + dk)[e & 3] = 0u;
  __syncthreads();
  // ---- causal matrix of the queries (to memory) and M (to shared memory): the 16 x 16 blocks on and below the diagonal
  __nv_bfloat16* am = reinterpret_cast<__nv_bfloat16*>(image + I.off_a);
  constexpr int NB = C / 16;
  const int gq = lane >> 2, t4 = lane & 3;
  if (fast) {
    for (int job = warp; job < 2 * NB * NB; job += 8) {  // (matrix, block)
      const bool is_m = job >= NB * NB;
      const int mb = (job % (NB * NB)) / NB, nb = job % NB;
      if (nb > mb) continue;
      float acc[2][4] = {};
      const uint32_t q_at = smem_u32((is_m ? sB : sQ) + (mb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * P + (lane >> 4) * 8);
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
          const int t = mb * 16 + gq + 8 * r, s = nb * 16 + n * 8 + 2 * t4;
          if (is_m) {
            sM[t * (C + 1) + s] = s < t ? acc[n][2 * r] * beta[t] : 0.f;
            sM[t * (C + 1) + s + 1] = s + 1 < t ? acc[n][2 * r + 1] * beta[t] : 0.f;
          } else {
            uint32_t hi, lw;
            split2(s <= t ? acc[n][2 * r] : 0.f, s + 1 <= t ? acc[n][2 * r + 1] : 0.f, hi, lw);
            *reinterpret_cast<uint32_t*>(am + t * I.PA + s) = hi;
            *reinterpret_cast<uint32_t*>(am + (C + t) * I.PA + s) = lw;
          }
        }
    }
  } else {
    for (int e = tid; e < C * C / 2; e += 256) {
      const int t = e / (C / 2), s = (e % (C / 2)) * 2;
      if (s / 16 > t / 16) continue;
      float v[2] = {0.f, 0.f}, m[2] = {0.f, 0.f};
      if (t < len) {
        const __nv_bfloat16* q = qp + static_cast<size_t>(t) * width;
        const __nv_bfloat16* kt = kp + static_cast<size_t>(t) * width;
        for (int j = 0; j < 2; ++j) {
          if (s + j > t) continue;
          const __nv_bfloat16* k = kp + static_cast<size_t>(s + j) * width;
          float acc = 0.f, accm = 0.f;
          for (int x = 0; x < dk; ++x) {
            const float kd = bf2f(k[x]) * dn_ex2(sb[t * dk + x] - sb[(s + j) * dk + x]);
            acc += bf2f(q[x]) * kd;
            accm += bf2f(kt[x]) * kd;
          }
          v[j] = acc * fq[t] * fk[s + j];
          m[j] = s + j < t ? accm * fk[t] * fk[s + j] * beta[t] : 0.f;
        }
      }
      uint32_t hi, lw;
      split2(v[0], v[1], hi, lw);
      *reinterpret_cast<uint32_t*>(am + t * I.PA + s) = hi;
      *reinterpret_cast<uint32_t*>(am + (C + t) * I.PA + s) = lw;
      sM[t * (C + 1) + s] = m[0];
      sM[t * (C + 1) + s + 1] = m[1];
    }
  }
  __syncthreads();
  // ---- X = (I + M)^-1: diagonal blocks by forward substitution (a thread keeps one column in registers), then the blocks below the diagonal,
  // X_ij = -X_ii sum_k M_ik X_kj
  constexpr int W = C + 1;
  if (tid < C) {
    const int blk = tid / 16, j = tid % 16;
    const float* m = sM + (blk * 16) * W + blk * 16;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) x[t] = t == j ? 1.f : 0.f;
#pragma unroll
    for (int s = 0; s < 15; ++s) {
#pragma unroll
      for (int t = s + 1; t < 16; ++t) x[t] -= m[t * W + s] * x[s];
    }
#pragma unroll
    for (int t = 0; t < 16; ++t) sX[(blk * 16 + t) * W + blk * 16 + j] = x[t];
  }
  __syncthreads();
  if constexpr (NB == 2) {
    const int t = tid >> 4, j = tid & 15;
    float y = 0.f;
#pragma unroll
    for (int s = 0; s < 16; ++s) y += sM[(16 + t) * W + s] * sX[s * W + j];
    __syncthreads();
    sM[(16 + t) * W + j] = y;  // (M's block is no longer needed)
    __syncthreads();
    y = 0.f;
#pragma unroll
    for (int s = 0; s < 16; ++s) y -= sX[(16 + t) * W + 16 + s] * sM[(16 + s) * W + j];
    sX[(16 + t) * W + j] = y;
    __syncthreads();
  }
  static_assert(NB <= 2, "blocks below the diagonal");
  for (int e = tid; e < C * C / 2; e += 256) {
    const int t = e / (C / 2), s = (e % (C / 2)) * 2;
    if (s / 16 > t / 16) continue;
    uint32_t hi, lw;
    split2(s <= t ? sX[t * W + s] * beta[s] : 0.f, s + 1 <= t ? sX[t * W + s + 1] * beta[s + 1] : 0.f, hi, lw);
    *reinterpret_cast<uint32_t*>(am + (2 * C + t) * I.PA + s) = hi;
    *reinterpret_cast<uint32_t*>(am + (3 * C + t) * I.PA + s) = lw;
  }
}

// A stage: the image of a chunk, then v [C][72].
template <int C, int NK>
struct DeltaStage {
  static constexpr int P = NK * 16 + 8, PV = kDnCols + 8, PA = C + 8;
  static constexpr int kA = DeltaImage<C>(NK).off_a, kDec = DeltaImage<C>(NK).off_dec, kV = DeltaImage<C>(NK).bytes;
  static constexpr int kBytes = (kV + C * PV * 2 + 127) / 128 * 128;
  static constexpr int PO = kDnCols + 4;
  static constexpr int kOut = 2 * kBytes;                        // both halves' shares of the outputs [2][C][PO]
  static constexpr int kR = kOut + 2 * C * PO * 4;               // shares of S^T K'^T: [8 warps][C / 2][32 lanes]
  static constexpr int kTotal = kR + 8 * (C / 2) * 32 * 4;
  static_assert(NK % 2 == 0 && kTotal <= 227 * 1024, "two stages must fit shared memory");
};

template <int C, int NK>
__global__ void __launch_bounds__(256, C == 16 && NK <= 8 ? 2 : 1) delta_chunks_kernel(const DeltaArgs a, const DeltaChunks c) {
  pdl_wait();
  pdl_trigger();
  using L = DeltaStage<C, NK>;
  constexpr int NH = NK / 2, NT = C / 8, KS = C / 16;  // 16-channel tiles per warp; 8- and 16-token tiles of a chunk
  extern __shared__ __align__(128) uint8_t dsm[];
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t4 = lane & 3, wd = warp & 3, hk = warp >> 2;  // 16 value columns, half of the key channels
  float* so = reinterpret_cast<float*>(dsm + L::kOut);
  float* sr = reinterpret_cast<float*>(dsm + L::kR);
  const int c0 = blockIdx.x * kDnCols, n_chunks = c.count[s], first = c.first[s];
  if (n_chunks == 0) return;
  const int dk = a.dk, dv = a.dv, width = 2 * a.G * dk + a.H * dv;
  const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.qkv) + 2 * a.G * dk + h * dv;
  float* state = a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * dk * dv;
  const bool fresh = a.positions[a.q_start[s]] == 0;

  auto load = [&](int i, int stage) {
    const int ck = first + i, row0 = c.row0[ck], len = c.len[ck];
    const uint32_t base = smem_u32(dsm + stage * L::kBytes);
    const uint8_t* image = static_cast<const uint8_t*>(c.images) + (static_cast<size_t>(ck) * a.H + h) * L::kV;
    for (int e = tid * 16; e < L::kV; e += 256 * 16) cp16(base + e, image + e, true);
    for (int e = tid; e < C * 8; e += 256) {
      const int t = e >> 3, x = (e & 7) * 8;
      const bool ok = t < len && c0 + x < dv;
      cp16(base + L::kV + (t * L::PV + x) * 2, vp + static_cast<size_t>(row0 + (ok ? t : 0)) * width + (ok ? c0 + x : 0), ok);
    }
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
    cp_wait<0>();
    __syncthreads();  // the chunk has arrived, and all warps are done with the one in front of it
    if (i + 1 < n_chunks) load(i + 1, (i + 1) & 1);
    const uint32_t base = smem_u32(dsm + (i & 1) * L::kBytes);
    const float* dec = reinterpret_cast<const float*>(dsm + (i & 1) * L::kBytes + L::kDec);
    const __nv_bfloat16* sv = reinterpret_cast<const __nv_bfloat16*>(dsm + (i & 1) * L::kBytes + L::kV);
    float o[NT][4], r[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
      r[j][0] = r[j][1] = r[j][2] = r[j][3] = 0.f;
    }
    // this half's share of S^T K'^T and of O^T = S^T Q^T
    const uint32_t q_at = base + (((lane & 7) + (lane >> 4) * 8) * L::P + hk * NH * 16 + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int kt = 0; kt < NH; ++kt) {
      uint32_t sh[4], sl[4];
      split2(st[2 * kt][0], st[2 * kt][1], sh[0], sl[0]);
      split2(st[2 * kt][2], st[2 * kt][3], sh[1], sl[1]);
      split2(st[2 * kt + 1][0], st[2 * kt + 1][1], sh[2], sl[2]);
      split2(st[2 * kt + 1][2], st[2 * kt + 1][3], sh[3], sl[3]);
#pragma unroll
      for (int np = 0; np < KS; ++np) {
        uint32_t b[4];
        ldm_x4(q_at + ((4 * C + np * 16) * L::P + kt * 16) * 2, b);
        mma16816(r[2 * np], sh, b[0], b[1]);
        mma16816(r[2 * np + 1], sh, b[2], b[3]);
        mma16816(r[2 * np], sl, b[0], b[1]);
        mma16816(r[2 * np + 1], sl, b[2], b[3]);
        ldm_x4(q_at + ((5 * C + np * 16) * L::P + kt * 16) * 2, b);
        mma16816(r[2 * np], sh, b[0], b[1]);
        mma16816(r[2 * np + 1], sh, b[2], b[3]);
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
    // the halves add their shares: V^T - S^T K'^T in both
    float* mine = sr + (warp * (C / 2)) * 32 + lane;
    const float* theirs = sr + ((warp ^ 4) * (C / 2)) * 32 + lane;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) mine[(j * 4 + e) * 32] = r[j][e];
    asm volatile("bar.sync %0, 64;" ::"r"(1 + wd) : "memory");
    uint32_t rh[KS][4], rl[KS][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        r[j][e] = bf2f(sv[(j * 8 + 2 * t4 + (e & 1)) * L::PV + wd * 16 + g + (e >> 1) * 8]) - (r[j][e] + theirs[(j * 4 + e) * 32]);
      split2(r[j][0], r[j][1], rh[j / 2][(j & 1) * 2], rl[j / 2][(j & 1) * 2]);
      split2(r[j][2], r[j][3], rh[j / 2][(j & 1) * 2 + 1], rl[j / 2][(j & 1) * 2 + 1]);
    }
    // U^T = R^T T^T
    float u[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) u[j][0] = u[j][1] = u[j][2] = u[j][3] = 0.f;
    const uint32_t a_at = base + L::kA + (((lane & 7) + (lane >> 4) * 8) * L::PA + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int np = ks; np < KS; ++np) {
        uint32_t b[4];
        ldm_x4(a_at + ((2 * C + np * 16) * L::PA + ks * 16) * 2, b);
        mma16816(u[2 * np], rh[ks], b[0], b[1]);
        mma16816(u[2 * np + 1], rh[ks], b[2], b[3]);
        mma16816(u[2 * np], rl[ks], b[0], b[1]);
        mma16816(u[2 * np + 1], rl[ks], b[2], b[3]);
        ldm_x4(a_at + ((3 * C + np * 16) * L::PA + ks * 16) * 2, b);
        mma16816(u[2 * np], rh[ks], b[0], b[1]);
        mma16816(u[2 * np + 1], rh[ks], b[2], b[3]);
      }
    uint32_t uh[KS][4], ul[KS][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      split2(u[j][0], u[j][1], uh[j / 2][(j & 1) * 2], ul[j / 2][(j & 1) * 2]);
      split2(u[j][2], u[j][3], uh[j / 2][(j & 1) * 2 + 1], ul[j / 2][(j & 1) * 2 + 1]);
    }
    // O^T += U^T A^T (the halves take every other block of tokens)
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      if ((ks & 1) != hk) continue;
#pragma unroll
      for (int np = ks; np < KS; ++np) {
        uint32_t b[4];
        ldm_x4(a_at + (np * 16 * L::PA + ks * 16) * 2, b);
        mma16816(o[2 * np], uh[ks], b[0], b[1]);
        mma16816(o[2 * np + 1], uh[ks], b[2], b[3]);
        mma16816(o[2 * np], ul[ks], b[0], b[1]);
        mma16816(o[2 * np + 1], ul[ks], b[2], b[3]);
        ldm_x4(a_at + ((C + np * 16) * L::PA + ks * 16) * 2, b);
        mma16816(o[2 * np], uh[ks], b[0], b[1]);
        mma16816(o[2 * np + 1], uh[ks], b[2], b[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) so[(hk * C + j * 8 + 2 * t4 + (e & 1)) * L::PO + wd * 16 + g + (e >> 1) * 8] = o[j][e];
    // S^T = S^T diag(decay) + U^T K
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
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int jp = 0; jp < NH; ++jp) {
        uint32_t b[4];
        ldm_x4_t(k_at + (ks * 16 * L::P + jp * 16) * 2, b);
        mma16816(st[2 * jp], uh[ks], b[0], b[1]);
        mma16816(st[2 * jp + 1], uh[ks], b[2], b[3]);
        mma16816(st[2 * jp], ul[ks], b[0], b[1]);
        mma16816(st[2 * jp + 1], ul[ks], b[2], b[3]);
        ldm_x4_t(k_at + ((C + ks * 16) * L::P + jp * 16) * 2, b);
        mma16816(st[2 * jp], uh[ks], b[0], b[1]);
        mma16816(st[2 * jp + 1], uh[ks], b[2], b[3]);
      }
    asm volatile("bar.sync %0, 64;" ::"r"(1 + wd) : "memory");  // both shares of these 16 columns are there
    const int row0 = c.row0[first + i], len = c.len[first + i];
#pragma unroll
    for (int e = hk * 32 + lane; e < C * 4; e += 64) {
      const int t = e >> 2, x = wd * 16 + (e & 3) * 4;
      if (t >= len || c0 + x >= dv) continue;
      const float4 p = *reinterpret_cast<const float4*>(so + t * L::PO + x), w = *reinterpret_cast<const float4*>(so + (C + t) * L::PO + x);
      *reinterpret_cast<float4*>(a.o + static_cast<size_t>(row0 + t) * (a.H * dv) + h * dv + c0 + x) = make_float4(p.x + w.x, p.y + w.y, p.z + w.z, p.w + w.w);
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
static cudaError_t launch_chunks_t(const DeltaArgs& a, const DeltaChunks& c, cudaStream_t st) {
  using L = DeltaStage<C, NK>;
  static PerDeviceOnce once;
  if (once.first()) {
    const cudaError_t e = cudaFuncSetAttribute(delta_chunks_kernel<C, NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kTotal);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(delta_chunks_kernel<C, NK>, dim3((a.dv + kDnCols - 1) / kDnCols, a.H, a.num_seqs), dim3(256), L::kTotal, st, a, c);
}

template <int C, int R>
static cudaError_t launch_prepare_t(const DeltaArgs& a, const DeltaChunks& c, cudaStream_t st) {
  const size_t smem = static_cast<size_t>(DeltaPrepareSmem<C, R>(a.dk).bytes);
  static PerDeviceOnce once;
  if (once.first()) {
    const cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<C, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(delta_prepare_kernel<C, R>, dim3(c.n_chunks, a.H), dim3(256), smem, st, a, c);
}

int launch_delta_chunked(const DeltaArgs& a, DeltaChunks c, cudaStream_t st) {
  if (a.rows == 0 || c.n_chunks == 0) return 0;
  c.tiles = delta_tiles(a.dk);
  cudaError_t e;
  if (c.chunk == 32 && a.dk <= 128) e = launch_prepare_t<32, 8>(a, c, st);
  else if (c.chunk == 16 && a.dk <= 128) e = launch_prepare_t<16, 4>(a, c, st);
  else if (c.chunk == 16 && a.dk <= 256) e = launch_prepare_t<16, 8>(a, c, st);
  else return 1;
  if (e == cudaSuccess) {
    if (c.chunk == 16) e = c.tiles == 16 ? launch_chunks_t<16, 16>(a, c, st) : c.tiles == 8 ? launch_chunks_t<16, 8>(a, c, st) : c.tiles == 4 ? launch_chunks_t<16, 4>(a, c, st) : launch_chunks_t<16, 2>(a, c, st);
    else e = c.tiles == 8 ? launch_chunks_t<32, 8>(a, c, st) : c.tiles == 4 ? launch_chunks_t<32, 4>(a, c, st) : launch_chunks_t<32, 2>(a, c, st);
  }
  if (e == cudaSuccess) e = launch_norm_gate(a, false, st);
  return e == cudaSuccess ? 0 : 2;
}

}  // namespace dlv
