// Several residual streams per token ("hyper-connections"): a sublayer reads a weighted sum of the streams and writes its output back to
// all of them while they are mixed among each other,
//   u = sum_s read[s] x_s,   x_t <- sum_s mix[s, t] x_s + write[t] y   (no new stream enters another one).
// stream_step_kernel finishes one sublayer and starts the next in a single pass over the fp32 streams X [T, S, W]:
//   y   one row of `sub`, or the weighted sum of k rows of an expert-ordered buffer (formed in fp32 in slot order),
//   X   rewritten (unless nothing reads it again),
//   out LayerNorm(sum_s read[s] x_s; w_next), weight without bias, columns W .. y_width zeroed.
// OPEN: the streams start here: X_s = LayerNorm(table[ids[t]]; w_open) for every s.
// One CTA per row; only the sum that the norm reads lives in registers (NV groups of four columns per thread).
#include "gemm_api.h"
#include "io.cuh"

namespace dlv {

template <typename TIO, int NV, int NT, int SMAX, bool OPEN>
__global__ void __launch_bounds__(NT) stream_step_kernel(const StreamArgs a) {
  __shared__ float red[32];
  const int t = blockIdx.x, W = a.W, S = a.S;
  float* X = a.streams + static_cast<size_t>(t) * S * W;
  TIO* y = static_cast<TIO*>(a.y) + t * a.ld_y;
  const TIO* sub = static_cast<const TIO*>(a.sub);
  auto col = [&](int n) { return (n * NT + static_cast<int>(threadIdx.x)) * 4; };
  auto load = [&](const auto* p, int c, float* o) {
    if (a.vec) {
      if (c < W) io_ld4(p + c, o);
      else o[0] = o[1] = o[2] = o[3] = 0.f;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = c + e < W ? io_ld(p + c + e) : 0.f;
    }
  };
  auto store = [&](float* p, int c, const float* v) {
    if (a.vec) {
      if (c < W) io_st4(p + c, v);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < W) p[c + e] = v[e];
    }
  };
  float v[NV][4];
  // mean of the real columns, and one over the root of the mean squared deviation from it
  auto statistics = [&](float& mean, float& inv) {
    float s = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) s += (v[n][0] + v[n][1]) + (v[n][2] + v[n][3]);
    mean = block_sum(s, red) / W;
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float d = v[n][e] - mean;
        ss += col(n) + e < W ? d * d : 0.f;
      }
    inv = rsqrtf(block_sum(ss, red) / W + a.eps);
  };
  // weights first: no kernel in front writes them, so their loads run under its tail
  float rd[SMAX], wr[SMAX], mix[SMAX <= 4 ? SMAX : 1][SMAX <= 4 ? SMAX : 1], wn[NV <= 4 ? NV : 1][4];
  const bool upd = !OPEN && sub != nullptr;
#pragma unroll
  for (int s = 0; s < SMAX; ++s) {
    rd[s] = s < S && a.read != nullptr ? a.read[s] : 1.f;
    wr[s] = upd && s < S ? a.write[s] : 0.f;
    if constexpr (SMAX <= 4 && !OPEN)
#pragma unroll
      for (int q = 0; q < SMAX; ++q) mix[s][q] = upd && s < S && q < S ? a.mix[s * S + q] : 0.f;
  }
  if constexpr (NV <= 4) {
    if (a.w_next != nullptr)
#pragma unroll
      for (int n = 0; n < NV; ++n) load(a.w_next, col(n), wn[n]);  // (zeros behind the row: so are the outputs there)
  }
  pdl_wait();
  pdl_trigger();
  if constexpr (OPEN) {
    int id = a.ids[t];
    if (id < 0 || id >= a.vocab) id = 0;  // host validates ids; never read out of the table
    sub += static_cast<size_t>(id) * a.ld_sub;
#pragma unroll
    for (int n = 0; n < NV; ++n) load(sub, col(n), v[n]);
    float mean, inv, total = 0.f;
    statistics(mean, inv);
#pragma unroll
    for (int s = 0; s < SMAX; ++s) total += s < S ? rd[s] : 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      float w[4];
      load(a.w_open, col(n), w);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[n][e] = (v[n][e] - mean) * inv * w[e];
      for (int s = 0; s < S; ++s) store(X + static_cast<size_t>(s) * W, col(n), v[n]);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[n][e] *= total;
    }
  } else {
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int c = col(n);
      float old[SMAX][4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int s = 0; s < SMAX; ++s)
        if (s < S) load(X + static_cast<size_t>(s) * W, c, old[s]);
        else old[s][0] = old[s][1] = old[s][2] = old[s][3] = 0.f;
      if (upd) {
        if (a.pos == nullptr) {
          load(sub + t * a.ld_sub, c, o);
        } else {
          for (int j = 0; j < a.k; ++j) {
            const float wt = a.wts[static_cast<size_t>(t) * a.k + j];
            float f[4];
            load(sub + a.pos[static_cast<size_t>(t) * a.k + j] * a.ld_sub, c, f);
#pragma unroll
            for (int e = 0; e < 4; ++e) o[e] += wt * f[e];
          }
        }
      }
      v[n][0] = v[n][1] = v[n][2] = v[n][3] = 0.f;
#pragma unroll
      for (int q = 0; q < SMAX; ++q) {
        if (q >= S) break;
        float x[4];
        if (upd) {
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = wr[q] * o[e];
#pragma unroll
          for (int s = 0; s < SMAX; ++s) {
            if (s >= S) break;
            float m;
            if constexpr (SMAX <= 4) m = mix[s][q];
            else m = a.mix[s * S + q];
#pragma unroll
            for (int e = 0; e < 4; ++e) x[e] = fmaf(m, old[s][e], x[e]);
          }
          if (a.keep) store(X + static_cast<size_t>(q) * W, c, x);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = old[q][e];
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) v[n][e] = fmaf(rd[q], x[e], v[n][e]);
      }
    }
  }
  float mean = 0.f, inv = 1.f;
  if (a.w_next != nullptr) statistics(mean, inv);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int c = col(n);
    float o[4] = {v[n][0], v[n][1], v[n][2], v[n][3]};
    if (a.w_next != nullptr) {
      float w[4];
      if constexpr (NV <= 4) {
#pragma unroll
        for (int e = 0; e < 4; ++e) w[e] = wn[n][e];
      } else {
        load(a.w_next, c, w);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = (o[e] - mean) * inv * w[e];
    }
    if (a.vec) {
      if (c < a.y_width) io_st4(y + c, o);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < a.y_width) io_st(y + c + e, o[e]);
    }
  }
}

template <typename TIO, int SMAX, bool OPEN>
static cudaError_t stream_dispatch(const StreamArgs& a, int rows, cudaStream_t st) {
  const int width = a.W > a.y_width ? a.W : a.y_width;
  if (width <= 512) return launch_pdl(stream_step_kernel<TIO, 1, 128, SMAX, OPEN>, dim3(rows), dim3(128), 0, st, a);
  if (width <= 1024) return launch_pdl(stream_step_kernel<TIO, 1, 256, SMAX, OPEN>, dim3(rows), dim3(256), 0, st, a);
  if (width <= 2048) return launch_pdl(stream_step_kernel<TIO, 2, 256, SMAX, OPEN>, dim3(rows), dim3(256), 0, st, a);
  if (width <= 4096) return launch_pdl(stream_step_kernel<TIO, 4, 256, SMAX, OPEN>, dim3(rows), dim3(256), 0, st, a);
  return launch_pdl(stream_step_kernel<TIO, 8, 512, SMAX, OPEN>, dim3(rows), dim3(512), 0, st, a);  // up to 16384 columns
}
template <typename TIO>
static cudaError_t stream_streams(const StreamArgs& a, int rows, cudaStream_t st) {
  if (a.ids != nullptr) return a.S <= 2 ? stream_dispatch<TIO, 2, true>(a, rows, st) : stream_dispatch<TIO, kMaxStreams, true>(a, rows, st);
  if (a.S <= 2) return stream_dispatch<TIO, 2, false>(a, rows, st);
  if (a.S <= 4) return stream_dispatch<TIO, 4, false>(a, rows, st);
  return stream_dispatch<TIO, kMaxStreams, false>(a, rows, st);
}

int launch_stream_step(const StreamArgs& a, int rows, bool is_f32, cudaStream_t st) {
  if (rows == 0) return 0;
  if (a.S < 1 || a.S > kMaxStreams || a.W < 1 || a.y_width > 16384 || a.W > 16384) return 1;
  return (is_f32 ? stream_streams<float>(a, rows, st) : stream_streams<__nv_bfloat16>(a, rows, st)) == cudaSuccess ? 0 : 2;
}

}  // namespace dlv
