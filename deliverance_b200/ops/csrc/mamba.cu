// Mamba-2 (state-space duality): per head  S_t = exp(neg_a dt_t) S_(t-1) + dt_t B_t x_t^T,  y_t = S_t^T C_t + D x_t  (S is dn x dv; heads of a group share B
// and C), dt = softplus(. + dt_bias); x, B and C come through a short convolution (short_conv.cu). The heads' columns are multiplied with silu(z) and
// RMS-normed in equal parts. State, dt, decays and everything that enters the recurrence besides projections and convolution are fp32.
//
//   mamba_recurrent_kernel  one CTA per (64 value columns, head, sequence), its part of the state in registers: decode steps (with the convolution of
//                           their token in the same launch, the ring of inputs updated in place), the 32-bit form of prompts, state sizes that the
//                           chunked form does not take.
//   mamba_dt_kernel         prompts, per (chunk, head): dt and the running sums of the base-2 log decays inside the chunk; the chunked form itself
//                           (contributions of all chunks, scan, outputs of all chunks) is that of lightning.cu with these decays.
//   mamba_norm_kernel       D x (chunked form), gate and norm.
// Reference of the granitemoehybrid layers (token by token): core/.../model/granitemoehybrid/GraniteMoeHybridMambaLayer.java:130-252.
#include "common.cuh"
#include "conv_step.cuh"
#include "gemm_api.h"
#include "io.cuh"

namespace dlv {

namespace {
constexpr int kMbCols = 64;  // value columns per CTA
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
}  // namespace

// 256 threads = 16 column groups (4 value columns each) x 16 row groups; thread (cx, rg) owns state rows rg, rg + 16, ..
template <typename TIO, int RPT, bool STEP>
__global__ void __launch_bounds__(256) mamba_recurrent_kernel(const MambaArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float sB[RPT * 16], sC[RPT * 16], sx[kMbCols];
  __shared__ float red[8][kMbCols];
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int cx = tid & 15, rg = tid >> 4, c_first = blockIdx.x * kMbCols, c0 = c_first + cx * 4;
  const bool col_ok = c0 < a.dv;
  const int row0 = a.q_start[s], n = a.q_len[s];
  if (n == 0) return;
  const int per_group = a.H / a.G, g = h / per_group;
  const int off_B = a.H * a.dv, off_C = off_B + a.G * a.dn, C = off_C + a.G * a.dn;  // columns of x | B | C
  const TIO* p = static_cast<const TIO*>(a.p);
  float* state = a.state + (static_cast<size_t>(a.slots[s]) * a.H + h) * a.dn * a.dv + c0;
  const int pos0 = a.positions[row0];
  const bool fresh = pos0 == 0;  // a sequence that starts at position 0 starts from a zero state
  const float neg_a = a.neg_a[h], dt_bias = a.dt_bias[h], D = a.D[h];
  float st[RPT][4];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + 16 * i;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh && col_ok && d < a.dn) v = *reinterpret_cast<const float4*>(state + static_cast<size_t>(d) * a.dv);
    st[i][0] = v.x; st[i][1] = v.y; st[i][2] = v.z; st[i][3] = v.w;
  }
  for (int t = 0; t < n; ++t) {
    const TIO* row = p + static_cast<size_t>(row0 + t) * a.ld;
    if constexpr (STEP) {
      // channels of this CTA: its value columns, B and C of its group (their ring rows are written by the group's first CTA)
      float* ring = a.ring + static_cast<size_t>(a.slots[s]) * a.taps * C;
      float* own = ring + static_cast<size_t>(pos0 % a.taps) * C;
      const TIO* in = row + a.H * a.dv;
      const bool writes = blockIdx.x == 0 && h % per_group == 0;
      for (int e = tid; e < 2 * RPT * 16 + kMbCols; e += 256) {
        if (e < 2 * RPT * 16) {
          const int d = e % (RPT * 16), c = (e < RPT * 16 ? off_B : off_C) + g * a.dn + d;
          float y = 0.f;
          if (d < a.dn) {
            const float x = io_ld(in + c);
            y = conv_step<TIO>(x, a.conv_w, a.conv_b, ring, a.taps, C, c, pos0);
            if (writes) own[c] = x;
          }
          (e < RPT * 16 ? sB : sC)[d] = y;
        } else {
          const int col = e - 2 * RPT * 16, c = h * a.dv + c_first + col;
          float y = 0.f;
          if (c_first + col < a.dv) {
            const float x = io_ld(in + c);
            y = conv_step<TIO>(x, a.conv_w, a.conv_b, ring, a.taps, C, c, pos0);
            own[c] = x;
          }
          sx[col] = y;
        }
      }
    } else {
      const TIO* in = static_cast<const TIO*>(a.xbc) + static_cast<size_t>(row0 + t) * C;
      for (int d = tid; d < RPT * 16; d += 256) {
        sB[d] = d < a.dn ? io_ld(in + off_B + g * a.dn + d) : 0.f;
        sC[d] = d < a.dn ? io_ld(in + off_C + g * a.dn + d) : 0.f;
      }
      if (tid < kMbCols) sx[tid] = c_first + tid < a.dv ? io_ld(in + h * a.dv + c_first + tid) : 0.f;
    }
    const float dt = softplus_f(io_ld(row + a.dt_at + h) + dt_bias), decay = expf(neg_a * dt);
    __syncthreads();
    float v[4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = sx[cx * 4 + e] * dt;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + 16 * i;
      const float k = sB[d], q = sC[d];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        st[i][e] = st[i][e] * decay + k * v[e];
        o[e] += st[i][e] * q;
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    if ((tid & 31) < 16) *reinterpret_cast<float4*>(&red[tid >> 5][cx * 4]) = make_float4(o[0], o[1], o[2], o[3]);
    const float xd = tid < kMbCols ? sx[tid] * D : 0.f;
    __syncthreads();  // (also: everyone is done with sB, sC and sx)
    if (tid < kMbCols) {
      float sum = xd;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[w][tid];
      const int c = c_first + tid;
      if (c < a.dv) a.y[static_cast<size_t>(row0 + t) * (a.H * a.dv) + h * a.dv + c] = sum;
    }
  }
  if (!col_ok) return;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + 16 * i;
    if (d < a.dn) *reinterpret_cast<float4*>(state + static_cast<size_t>(d) * a.dv) = make_float4(st[i][0], st[i][1], st[i][2], st[i][3]);
  }
}

// grid (rows, norm groups): y (+ D x with xbc) times silu(z), RMS norm over the group's real columns, weight
template <typename TIO, bool ADD_X>
__global__ void __launch_bounds__(256) mamba_norm_kernel(const MambaArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  constexpr int KEEP = 8;  // four-column pieces a thread keeps between the two passes
  const int t = blockIdx.x, n = a.H * a.dv_real / a.norm_groups, first = blockIdx.y * n;
  const float* y = a.y + static_cast<size_t>(t) * (a.H * a.dv);
  const TIO* z = static_cast<const TIO*>(a.p) + static_cast<size_t>(t) * a.ld;
  const TIO* x = ADD_X ? static_cast<const TIO*>(a.xbc) + static_cast<size_t>(t) * (a.H * a.dv + 2 * a.G * a.dn) : nullptr;
  TIO* out = static_cast<TIO*>(a.out) + static_cast<size_t>(t) * (a.H * a.dv);
  if (a.dv == a.dv_real && n % 4 == 0) {
    auto gated = [&](int c, float* v) {
      float zv[4];
      io_ld4(y + c, v);
      io_ld4(z + c, zv);
      if constexpr (ADD_X) {
        float xv[4];
        io_ld4(x + c, xv);
        const float D = a.D[c / a.dv];  // (head widths are multiples of 8)
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] += D * xv[e];
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] *= zv[e] / (1.f + __expf(-zv[e]));
    };
    float keep[KEEP][4], ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * blockDim.x + threadIdx.x) * 4;
      if (c < n) {
        gated(first + c, keep[k]);
#pragma unroll
        for (int e = 0; e < 4; ++e) ss += keep[k][e] * keep[k][e];
      }
    }
    for (int c = (KEEP * blockDim.x + threadIdx.x) * 4; c < n; c += blockDim.x * 4) {
      float v[4];
      gated(first + c, v);
#pragma unroll
      for (int e = 0; e < 4; ++e) ss += v[e] * v[e];
    }
    const float inv = rsqrtf(block_sum(ss, red) / n + a.eps);
    auto put = [&](int c, float* v) {
      float w[4];
      io_ld4(a.norm_w + c, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] *= inv * w[e];
      io_st4(out + c, v);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * blockDim.x + threadIdx.x) * 4;
      if (c < n) put(first + c, keep[k]);
    }
    for (int c = (KEEP * blockDim.x + threadIdx.x) * 4; c < n; c += blockDim.x * 4) {
      float v[4];
      gated(first + c, v);
      put(first + c, v);
    }
    return;
  }
  auto gated1 = [&](int r, int& c) {  // real column r of the row, its place c in the padded layout
    const int h = r / a.dv_real;
    c = h * a.dv + r % a.dv_real;
    float v = y[c];
    if constexpr (ADD_X) v += a.D[h] * io_ld(x + c);
    const float zv = io_ld(z + c);
    return v * zv / (1.f + __expf(-zv));
  };
  float ss = 0.f;
  int c;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = gated1(first + i, c);
    ss += v * v;
  }
  const float inv = rsqrtf(block_sum(ss, red) / n + a.eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = gated1(first + i, c);
    io_st(out + c, v * inv * a.norm_w[c]);
  }
}

template <typename TIO, bool ADD_X>
static cudaError_t launch_norm_t(const MambaArgs& a, cudaStream_t st) {
  const int n = a.H * a.dv_real / a.norm_groups, threads = n >= 4096 ? 256 : (n >= 512 ? 128 : 64);
  return launch_pdl(mamba_norm_kernel<TIO, ADD_X>, dim3(a.rows, a.norm_groups), dim3(threads), 0, st, a);
}

template <typename TIO, bool STEP>
static cudaError_t launch_recurrent_t(const MambaArgs& a, cudaStream_t st) {
  const dim3 grid((a.dv + kMbCols - 1) / kMbCols, a.H, a.num_seqs);
  if (a.dn <= 32) return launch_pdl(mamba_recurrent_kernel<TIO, 2, STEP>, grid, dim3(256), 0, st, a);
  if (a.dn <= 64) return launch_pdl(mamba_recurrent_kernel<TIO, 4, STEP>, grid, dim3(256), 0, st, a);
  if (a.dn <= 128) return launch_pdl(mamba_recurrent_kernel<TIO, 8, STEP>, grid, dim3(256), 0, st, a);
  if (a.dn <= 256) return launch_pdl(mamba_recurrent_kernel<TIO, 16, STEP>, grid, dim3(256), 0, st, a);
  return launch_pdl(mamba_recurrent_kernel<TIO, 32, STEP>, grid, dim3(256), 0, st, a);
}

int launch_mamba2_recurrent(const MambaArgs& a, bool is_f32, cudaStream_t st) {
  if (a.rows == 0 || a.num_seqs == 0) return 0;
  const bool step = a.xbc == nullptr;
  if (a.dn > 512 || (step && (a.rows != a.num_seqs || a.taps < 1))) return 1;
  cudaError_t e;
  if (is_f32) e = step ? launch_recurrent_t<float, true>(a, st) : launch_recurrent_t<float, false>(a, st);
  else e = step ? launch_recurrent_t<__nv_bfloat16, true>(a, st) : launch_recurrent_t<__nv_bfloat16, false>(a, st);
  if (e == cudaSuccess) e = is_f32 ? launch_norm_t<float, false>(a, st) : launch_norm_t<__nv_bfloat16, false>(a, st);
  return e == cudaSuccess ? 0 : 2;
}

// one warp per (chunk, head), four tokens per lane
__global__ void __launch_bounds__(256) mamba_dt_kernel(const MambaArgs a, const LightningChunks c, int chunk) {
  pdl_wait();
  pdl_trigger();
  const int ck = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= a.H) return;
  const int row0 = c.row0[ck], len = c.len[ck];
  const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(a.p) + a.dt_at + h;
  const float scale = a.neg_a[h] * 1.4426950408889634f, bias = a.dt_bias[h];
  float carry = 0.f;
  for (int t0 = 0; t0 < chunk; t0 += 128) {
    float dt[4], sum = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = t0 + lane * 4 + i;
      dt[i] = t < len ? softplus_f(bf2f(p[static_cast<size_t>(row0 + t) * a.ld]) + bias) : 0.f;
      sum += dt[i];
    }
    float before = sum;  // inclusive scan over the lanes
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += up;
    }
    const float total = __shfl_sync(0xffffffffu, before, 31);
    before -= sum;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = t0 + lane * 4 + i;
      before += dt[i];
      if (t < len) {
        const size_t at = static_cast<size_t>(row0 + t) * a.H + h;
        a.dt[at] = dt[i];
        a.cum[at] = (carry + before) * scale;
      }
    }
    carry += total;
  }
}

int launch_mamba2_chunked(const MambaArgs& a, const LightningChunks& c, int chunk, cudaStream_t st) {
  if (a.rows == 0 || c.n_chunks == 0) return 0;
  if (a.xbc == nullptr || chunk % 128 != 0) return 1;
  if (launch_pdl(mamba_dt_kernel, dim3(c.n_chunks, (a.H + 7) / 8), dim3(256), 0, st, a, c, chunk) != cudaSuccess) return 2;
  LightningArgs l = {};
  l.p = a.xbc;
  l.ld = a.H * a.dv + 2 * a.G * a.dn;
  l.H = a.H;
  l.dk = a.dn;
  l.dv = a.dv;
  l.off_v = 0;
  l.off_k = a.H * a.dv;
  l.off_q = l.off_k + a.G * a.dn;
  l.qk_div = a.H / a.G;
  l.cum = a.cum;
  l.vscale = a.dt;
  l.chunk = chunk;
  l.state = a.state;
  l.slots = a.slots;
  l.q_start = a.q_start;
  l.q_len = a.q_len;
  l.positions = a.positions;
  l.num_seqs = a.num_seqs;
  l.rows = a.rows;
  l.o = a.y;
  const int rc = launch_decayed_chunks(l, c, st);
  if (rc != 0) return rc;
  return launch_norm_t<__nv_bfloat16, true>(a, st) == cudaSuccess ? 0 : 2;
}

}  // namespace dlv
