// Softmax attention whose heads' scores are mixed by a matrix in front of the softmax:  score_h = scale sum_g mix[h, g] (q_g . k_(g's KV head)).
// Cache rows are wide: k [pages, 1, page, KV dk] and v [pages, 1, page, KV dv] hold all KV heads of a token side by side.
//
//   mixed_decode_kernel  decode, grid (splits, sequences): one CTA takes ALL heads of a row. Tiles of 32 keys arrive by cp.async; per tile: raw scores of every
//                        head on mma.sync (the heads of a KV head are the rows of the operand), through shared memory to the mixing and the online softmax
//                        in fp32 (a warp owns heads, a lane a key), and back as the bf16 operand of the weighted sums, for which the warps split the value
//                        columns of all KV heads. The splits of a row are merged by the merge kernel of the grouped decode attention.
//   fold_heads_kernel    prompts and the 32-bit form: the mixing moves to the query side, q'[h] = [sum_(g of KV head 0) mix[h, g] q_g | .. of KV head 1 | ..], so
//                        that a head's mixed score is one product with the whole cache row (attention_tc.cu, wide rows; attn_rows_kernel).
#include "common.cuh"
#include "gemm_api.h"
#include "io.cuh"
#include "mma_pair.cuh"

namespace dlv {

constexpr int kMxBK = 32;       // keys per tile
constexpr int kMxHeads = 64;    // most query heads
constexpr int kMxBlocks = 8;    // most 16-column value blocks per warp

struct MixedDecodeSmem {
  int pk, pv, pq, stages;  // row pitches (elements) of keys, values and queries
  int off_v, stage, off_q, off_p, off_s, off_m, off_st, bytes;
  static constexpr int kPP = kMxBK + 8, kPS = kMxBK + 1;
  static __host__ __device__ int pitch(int w) { return w + ((w / 8) % 2 == 0 ? 8 : 16); }  // odd in units of 16 bytes, at least 8 columns to spare
  __host__ __device__ MixedDecodeSmem(int H, int KV, int dk, int dv, int n_stages) {
    pk = pitch(KV * dk);
    pv = pitch(KV * dv);
    pq = (dk + 15) / 16 * 16 + 8;
    stages = n_stages;
    off_v = kMxBK * pk * 2;
    stage = off_v + kMxBK * pv * 2;
    off_q = stages * stage;
    off_p = off_q + (H + 1) * pq * 2;   // (one row of zeros behind the heads)
    off_s = off_p + (H + 1) * kPP * 2;
    off_m = off_s + H * kPS * 4;
    off_st = off_m + H * H * 4;
    bytes = off_st + 2 * (H + 1) * 4;
  }
};

static int mixed_stages(int H, int KV, int dk, int dv) {
  for (int n = 3; n >= 1; --n)
    if (MixedDecodeSmem(H, KV, dk, dv, n).bytes <= 227 * 1024) return n;
  return 0;
}
static int mixed_blocks(int H, int KV, int dv) {  // 16-column value blocks per warp
  const int mt = (H / KV + 15) / 16;
  return (KV * mt * ((dv + 15) / 16) + 7) / 8;
}
bool mixed_decode_supported(int H, int KV, int dk, int dv) {
  return H >= 1 && H <= kMxHeads && H % KV == 0 && dk % 8 == 0 && dv % 8 == 0 && dk > 0 && dv > 0 && mixed_blocks(H, KV, dv) <= kMxBlocks &&
         mixed_stages(H, KV, dk, dv) > 0;
}

template <int NB>
__global__ void __launch_bounds__(256, 1) mixed_decode_kernel(const MixedDecodeArgs a, int stages) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t msm[];
  const MixedDecodeSmem L(a.H, a.KV, a.dk, a.dv, stages);
  constexpr int BK = kMxBK, PP = MixedDecodeSmem::kPP, PS = MixedDecodeSmem::kPS, HPW = kMxHeads / 8;
  const int H = a.H, dk = a.dk, dv = a.dv, per = H / a.KV, MT = (per + 15) / 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, t4 = lane & 3;
  const int b = blockIdx.y, sp = blockIdx.x, splits = gridDim.x;
  const uint32_t base = smem_u32(msm);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(msm + L.off_q);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(msm + L.off_p);
  float* sS = reinterpret_cast<float*>(msm + L.off_s);
  float* sM = reinterpret_cast<float*>(msm + L.off_m);
  float* sA = reinterpret_cast<float*>(msm + L.off_st);  // [H + 1] factor of the accumulators
  float* sF = sA + H + 1;                                // [H + 1] final factor
  const int ctx = a.ctx[b], first_key = (a.window > 0 && ctx > a.window) ? ctx - a.window : 0;
  const int tl = first_key / BK, th = (ctx + BK - 1) / BK, per_split = (th - tl + splits - 1) / splits;
  const int t0 = tl + sp * per_split, nt = max(0, min(th, t0 + per_split) - t0);
  const int* table = a.bt + static_cast<long long>(b) * a.bt_stride;
  const int wk = a.KV * dk, wv = a.KV * dv;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(a.kc);
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.vc);

  // a warp copies rows warp, warp + 8, .. of a tile (a tile lies inside one page; rows behind the context are rows of the same page: finite
  // values that the mask gives weight zero)
  auto load = [&](int j) {
    const int key0 = (t0 + j) * BK;
    const long long row0 = static_cast<long long>(table[key0 / a.page]) * a.page + key0 % a.page;
    const uint32_t dst = base + (j % stages) * L.stage;
    for (int r = warp; r < BK; r += 8) {
      const __nv_bfloat16* k = kc + (row0 + r) * wk;
      const __nv_bfloat16* v = vc + (row0 + r) * wv;
      for (int x = lane * 8; x < wk; x += 256) cp16(dst + (r * L.pk + x) * 2, k + x, true);
      for (int x = lane * 8; x < wv; x += 256) cp16(dst + L.off_v + (r * L.pv + x) * 2, v + x, true);
    }
  };
  for (int j = 0; j < max(1, stages - 1); ++j) {
    if (j < nt) load(j);
    cp_commit();
  }
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + b * a.q_stride;
  for (int e = tid; e < (H + 1) * (L.pq / 8); e += 256) {
    const int r = e / (L.pq / 8), x = (e % (L.pq / 8)) * 8;
    *reinterpret_cast<uint4*>(sQ + r * L.pq + x) = r < H && x < dk ? *reinterpret_cast<const uint4*>(q + r * dk + x) : make_uint4(0u, 0u, 0u, 0u);
  }
  for (int e = tid; e < H * H; e += 256) sM[e] = a.mix[e] * a.scale;
  for (int e = tid; e < PP; e += 256) sP[H * PP + e] = f2bf(0.f);
  if (tid == 0) sA[H] = 1.f;
  // columns behind a key row meet zero queries: they must be finite
  for (int e = tid; e < stages * BK; e += 256)
    *reinterpret_cast<uint4*>(msm + (e / BK) * L.stage + ((e % BK) * L.pk + wk) * 2) = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();

  float m_run[HPW], l_run[HPW];  // softmax state of heads warp, warp + 8, ..; the sum is a part per lane
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
  }
  float o[NB][2][4];
  int ha[NB], hb[NB], hp[NB], vcol[NB];  // per value block: heads of rows gq and gq + 8 of the operand, of this lane's operand row (H: none), first column
  const int dvb = (dv + 15) / 16, blocks = a.KV * MT * dvb;
#pragma unroll
  for (int i = 0; i < NB; ++i) {
    const int blk = warp + 8 * i, m = blk / dvb, kvh = m / MT, h0 = (m % MT) * 16;
    auto head = [&](int r) { return blk < blocks && h0 + r < per ? kvh * per + h0 + r : H; };
    ha[i] = head(gq);
    hb[i] = head(gq + 8);
    hp[i] = head(lane & 15);
    vcol[i] = blk < blocks ? kvh * dv + (blk % dvb) * 16 : -1;
#pragma unroll
    for (int n = 0; n < 2; ++n) o[i][n][0] = o[i][n][1] = o[i][n][2] = o[i][n][3] = 0.f;
  }
  const int nks = (dk + 15) / 16, tasks = a.KV * MT * (BK / 8);
  for (int it = 0; it < nt; ++it) {
    if (stages == 3) cp_wait<1>();
    else cp_wait<0>();
    __syncthreads();  // the tile is here, and every warp is done with the stage of the previous one
    if (stages > 1) {
      if (it + stages - 1 < nt) load(it + stages - 1);
      cp_commit();
    }
    const uint32_t st = base + (it % stages) * L.stage;
    // ---- raw scores of every head
    for (int task = warp; task < tasks; task += 8) {
      const int kb = task % (BK / 8), m = task / (BK / 8), kvh = m / MT, h0 = (m % MT) * 16;
      const int hr = h0 + (lane & 15) < per ? kvh * per + h0 + (lane & 15) : H;
      const uint32_t qa = smem_u32(sQ + hr * L.pq + (lane >> 4) * 8);
      const uint32_t ka = st + ((kb * 8 + (lane & 7)) * L.pk + kvh * dk + (lane >> 3) * 8) * 2;  // two k16 steps per ldmatrix
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      int k = 0;
      for (; k + 1 < nks; k += 2) {
        uint32_t a0[4], a1[4], kb4[4];
        ldm_x4(ka + k * 32, kb4);
        ldm_x4(qa + k * 32, a0);
        ldm_x4(qa + k * 32 + 32, a1);
        mma16816(s0, a0, kb4[0], kb4[1]);
        mma16816(s1, a1, kb4[2], kb4[3]);
      }
      if (k < nks) {  // one step: lanes 16.. repeat the addresses of lanes 0..
        uint32_t a0[4], kb4[4];
        ldm_x4(ka + k * 32 - ((lane >> 4) << 5), kb4);
        ldm_x4(qa + k * 32, a0);
        mma16816(s0, a0, kb4[0], kb4[1]);
      }
      const int key = kb * 8 + 2 * t4, ra = h0 + gq, rb = ra + 8;
      if (ra < per) {
        sS[(kvh * per + ra) * PS + key] = s0[0] + s1[0];
        sS[(kvh * per + ra) * PS + key + 1] = s0[1] + s1[1];
      }
      if (rb < per) {
        sS[(kvh * per + rb) * PS + key] = s0[2] + s1[2];
        sS[(kvh * per + rb) * PS + key + 1] = s0[3] + s1[3];
      }
    }
    __syncthreads();
    // ---- mixing and online softmax. The running maximum follows only when a score has outgrown it by more than 8.
    const int key = (t0 + it) * BK + lane;
    const bool visible = key < ctx && key >= first_key;
    bool grown = false;
#pragma unroll
    for (int i = 0; i < HPW; ++i) {
      const int h = warp + 8 * i;
      if (h < H) {  // warp-uniform
        float v = 0.f;
        const float* mh = sM + h * H;
#pragma unroll 4
        for (int g = 0; g < H; ++g) v += mh[g] * sS[g * PS + lane];
        if (!visible) v = -INFINITY;
        float alpha = 1.f;
        if (__any_sync(0xffffffffu, v > m_run[i] + 8.f)) {
          const float mx = fmaxf(m_run[i], warp_max(v));
          alpha = __expf(m_run[i] - mx);  // (exp of -infinity: 0)
          m_run[i] = mx;
          l_run[i] *= alpha;
          grown = true;
        }
        const float p = v == -INFINITY ? 0.f : __expf(v - m_run[i]);
        l_run[i] += p;
        sP[h * PP + lane] = f2bf(p);
        if (lane == 0) sA[h] = alpha;
      }
    }
    const bool rescale = __syncthreads_or(grown);
    // ---- weighted sums: warp w owns the 16-column blocks w, w + 8, ..
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      if (vcol[i] < 0) continue;  // warp-uniform
      if (rescale) {
        const float fa = sA[ha[i]], fb = sA[hb[i]];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          o[i][n][0] *= fa;
          o[i][n][1] *= fa;
          o[i][n][2] *= fb;
          o[i][n][3] *= fb;
        }
      }
      const uint32_t pa = smem_u32(sP + hp[i] * PP + (lane >> 4) * 8);
      const uint32_t va = st + L.off_v + (((lane & 7) + ((lane >> 3) & 1) * 8) * L.pv + vcol[i] + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int ks = 0; ks < BK / 16; ++ks) {
        uint32_t p4[4], v4[4];
        ldm_x4(pa + ks * 32, p4);
        ldm_x4_t(va + ks * 16 * L.pv * 2, v4);
        mma16816(o[i][0], p4, v4[0], v4[1]);
        mma16816(o[i][1], p4, v4[2], v4[3]);
      }
    }
    if (stages == 1) {
      __syncthreads();
      if (it + 1 < nt) load(it + 1);
      cp_commit();
    }
  }
  cp_wait<0>();
  // ---- out
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int h = warp + 8 * i;
    if (h < H) {
      const float l = warp_sum(l_run[i]);
      if (lane == 0) {
        if (splits > 1) {
          float* ml = a.part_ml + ((static_cast<size_t>(b) * H + h) * splits + sp) * 2;
          ml[0] = m_run[i];
          ml[1] = l;
        } else {
          float f = l > 0.f ? a.x.out_mult / l : 0.f;
          if (a.x.gate != nullptr) f /= 1.f + expf(-bf2f(static_cast<const __nv_bfloat16*>(a.x.gate)[b * a.x.gate_pitch + h]));
          sF[h] = f;
        }
      }
    }
  }
  __syncthreads();
  const long long pitch = a.x.out_pitch > 0 ? a.x.out_pitch : static_cast<long long>(H) * dv;
#pragma unroll
  for (int i = 0; i < NB; ++i) {
    if (vcol[i] < 0) continue;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int h = half ? hb[i] : ha[i];
      if (h >= H) continue;
      const int c0 = vcol[i] % dv;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int c = c0 + n * 8 + 2 * t4;
        if (c >= dv) continue;
        const float x = o[i][n][half * 2], y = o[i][n][half * 2 + 1];
        if (splits > 1) {
          *reinterpret_cast<float2*>(a.part_o + ((static_cast<size_t>(b) * H + h) * splits + sp) * dv + c) = make_float2(x, y);
        } else {
          const float f = sF[h];
          *reinterpret_cast<uint32_t*>(static_cast<__nv_bfloat16*>(a.out) + b * pitch + h * dv + c) = pack_bf162(x * f, y * f);
        }
      }
    }
  }
}

template <int NB>
static int launch_mixed_decode_t(const MixedDecodeArgs& a, cudaStream_t st) {
  const int stages = mixed_stages(a.H, a.KV, a.dk, a.dv);
  static PerDeviceOnce once;
  if (once.first() && cudaFuncSetAttribute(mixed_decode_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return 2;
  const size_t smem = static_cast<size_t>(MixedDecodeSmem(a.H, a.KV, a.dk, a.dv, stages).bytes);
  if (launch_pdl(mixed_decode_kernel<NB>, dim3(a.splits, a.B), dim3(256), smem, st, a, stages) != cudaSuccess) return 2;
  if (a.splits > 1) launch_decode_merge(a.part_o, a.part_ml, a.out, a.B, a.H, a.dv, a.splits, a.x, st);
  return 0;
}

int launch_mixed_decode(const MixedDecodeArgs& a, cudaStream_t st) {
  if (a.B == 0) return 0;
  if (!mixed_decode_supported(a.H, a.KV, a.dk, a.dv) || a.page % kMxBK != 0 || a.q_stride % 8 != 0 || a.B > 65535 || a.splits < 1 || a.x.sink != nullptr ||
      (a.x.gate != nullptr && !a.x.gate_heads))
    return 1;
  const int nb = mixed_blocks(a.H, a.KV, a.dv);
  if (nb <= 1) return launch_mixed_decode_t<1>(a, st);
  if (nb <= 2) return launch_mixed_decode_t<2>(a, st);
  if (nb <= 4) return launch_mixed_decode_t<4>(a, st);
  return launch_mixed_decode_t<8>(a, st);
}

// out [T, H, KV dk]: a thread takes eight columns of one (row, head, KV head)
template <typename TIO>
__global__ void __launch_bounds__(256) fold_heads_kernel(const TIO* __restrict__ q, long long q_stride, const float* __restrict__ mix, TIO* __restrict__ out, int H,
                                                         int KV, int dk, long long total) {
  pdl_wait();
  pdl_trigger();
  const long long idx = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (idx >= total) return;
  const int vecs = dk / 8, x = static_cast<int>(idx % vecs) * 8, per = H / KV;
  const long long i = idx / vecs;
  const int kvh = static_cast<int>(i % KV), h = static_cast<int>((i / KV) % H);
  const long long t = i / KV / H;
  const TIO* src = q + t * q_stride + static_cast<long long>(kvh * per) * dk + x;
  const float* m = mix + h * H + kvh * per;
  float acc[8] = {};
#pragma unroll 4
  for (int g = 0; g < per; ++g) {
    float v[8];
    io_ld8(src + g * dk, v);
    const float w = m[g];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] += w * v[e];
  }
  io_st8(out + i * dk + x, acc);
}

void launch_fold_heads(const void* q, long long q_stride, const float* mix, void* out, int T, int H, int KV, int dk, bool is_f32, cudaStream_t st) {
  const long long total = static_cast<long long>(T) * H * KV * (dk / 8);
  if (total == 0) return;
  const dim3 grid(static_cast<unsigned>((total + 255) / 256));
  if (is_f32) launch_pdl(fold_heads_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(q), q_stride, mix, static_cast<float*>(out), H, KV, dk, total);
  else
    launch_pdl(fold_heads_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(q), q_stride, mix, static_cast<__nv_bfloat16*>(out), H, KV,
               dk, total);
}

}  // namespace dlv
