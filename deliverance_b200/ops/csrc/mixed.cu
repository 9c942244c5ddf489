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
constexpr int kMxBlocks = 8;    // most 16-column value blocks per warp (of eight)

struct MixedDecodeSmem {
  int pk, pv, pq, stages;  // row pitches (elements) of keys, values and queries
  int off_v, stage, off_q, off_p, off_s, off_m, off_st, bytes;
  static constexpr int kPP = kMxBK + 8, kPS = kMxBK + 1;
  static __host__ __device__ int pitch(int w) { return w + ((w / 8) % 2 == 0 ? 8 : 16); }  // odd in units of 16 bytes, at least 8 columns to spare
  __host__ __device__ MixedDecodeSmem(int H, int KV, int dk, int dv, int n_stages, int mix_heads) {
    pk = pitch(KV * dk);
    pv = pitch(KV * dv);
    pq = (dk + 15) / 16 * 16 + 8;
    stages = n_stages;
    off_v = kMxBK * pk * 2;
    stage = off_v + kMxBK * pv * 2;
    off_q = stages * stage;
    off_p = off_q + (H + 1) * pq * 2;   // (one row of zeros behind the heads)
    off_s = off_p + (H + 1) * kPP * 2;
    off_m = (off_s + H * kPS * 4 + 15) / 16 * 16;
    off_st = off_m + H * mix_heads * 4; // [H][mix_heads]: the matrix by source head, target heads in the order of the warps
    bytes = off_st + 2 * (H + 1) * 4;
  }
};

// How a shape runs: warps per CTA, heads per warp (the mixing), value blocks per warp, score tasks (KV head, group of 16 query heads, 8 keys) per warp whose
// queries stay in registers (0: any number, queries from shared memory) and their 16-column steps, stages and CTAs per SM.
struct MixedPlan {
  int warps, hpw, blocks, tasks, steps, stages, ctas;
};
static MixedPlan mixed_plan(int H, int KV, int dk, int dv) {
  MixedPlan p = {};
  if (H < 1 || H > kMxHeads || KV < 1 || H % KV != 0 || dk <= 0 || dv <= 0 || dk % 8 != 0 || dv % 8 != 0) return p;
  const int groups = KV * ((H / KV + 15) / 16), blocks = groups * ((dv + 15) / 16);
  auto bytes = [&](int stages, int warps, int hpw) { return MixedDecodeSmem(H, KV, dk, dv, stages, warps * hpw).bytes; };
  auto up = [](int n) { return n <= 2 ? 2 : (n <= 4 ? 4 : 8); };
  const int two = 113 * 1024, one = 227 * 1024;
  if (groups * ((dk + 63) / 64) <= 4 && dk <= 128 && H <= 32 && (blocks + 7) / 8 <= 4 && bytes(2, 8, up((H + 7) / 8)) <= two) {
    const int steps = dk <= 64 ? 4 : 8;
    p = {8, up((H + 7) / 8), up((blocks + 7) / 8), 8 / steps, steps, 2, 2};
  } else if (dk <= 128 && groups <= 8 && (blocks + 15) / 16 <= 4 && bytes(2, 16, up((H + 15) / 16)) <= one) {
    p = {16, up((H + 15) / 16), up((blocks + 15) / 16), groups <= 4 ? 1 : 2, 8, 2, 1};
    if (bytes(3, 16, p.hpw) <= one) p.stages = 3;
  } else if ((blocks + 7) / 8 <= kMxBlocks) {
    p = {8, 8, up((blocks + 7) / 8), 0, 0, 0, 1};
    for (int n = 3; n >= 1 && p.stages == 0; --n)
      if (bytes(n, 8, 8) <= one) p.stages = n;
    if (p.stages == 0) p.warps = 0;
  }
  return p;
}
bool mixed_decode_supported(int H, int KV, int dk, int dv) { return mixed_plan(H, KV, dk, dv).warps > 0; }
int mixed_decode_ctas(int H, int KV, int dk, int dv) { return mixed_plan(H, KV, dk, dv).ctas; }

template <int NW, int HPW, int NB, int NTK, int NQ>
__global__ void __launch_bounds__(NW * 32, NTK > 0 && NW == 8 ? 2 : 1) mixed_decode_kernel(const MixedDecodeArgs a, int stages) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t msm[];
  const MixedDecodeSmem L(a.H, a.KV, a.dk, a.dv, stages, NW * HPW);
  constexpr int BK = kMxBK, PP = MixedDecodeSmem::kPP, PS = MixedDecodeSmem::kPS, NT = NW * 32;
  const int H = a.H, dk = a.dk, dv = a.dv, per = H / a.KV, MT = (per + 15) / 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, t4 = lane & 3;
  const int b = blockIdx.y, sp = blockIdx.x, splits = gridDim.x;
  const uint32_t base = smem_u32(msm);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(msm + L.off_q);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(msm + L.off_p);
  float* sS = reinterpret_cast<float*>(msm + L.off_s);
  float* sM = reinterpret_cast<float*>(msm + L.off_m);   // [source head][warp][HPW]
  float* sA = reinterpret_cast<float*>(msm + L.off_st);  // [H + 1] factor of the accumulators
  float* sF = sA + H + 1;                                // [H + 1] final factor
  const int ctx = a.ctx[b], first_key = (a.window > 0 && ctx > a.window) ? ctx - a.window : 0;
  const int tl = first_key / BK, th = (ctx + BK - 1) / BK, per_split = (th - tl + splits - 1) / splits;
  const int t0 = tl + sp * per_split, nt = max(0, min(th, t0 + per_split) - t0);
  const int* table = a.bt + static_cast<long long>(b) * a.bt_stride;
  const int wk = a.KV * dk, wv = a.KV * dv;

  // A warp copies rows warp, warp + NW, .. of a tile. A tile lies inside one page; rows behind the context are rows of the same page: finite values that
  // the mask gives weight zero. The place of the next tile (page index, its id, first row in it) is known one tile ahead.
  int pidx = t0 * BK / a.page, poff = t0 * BK - pidx * a.page, pg = nt > 0 ? table[pidx] : 0;
  const char* kbase = reinterpret_cast<const char*>(a.kc) + lane * 16;
  const char* vbase = reinterpret_cast<const char*>(a.vc) + lane * 16;
  auto load = [&](int j) {
    const unsigned row0 = static_cast<unsigned>(pg) * a.page + poff + warp;
    const uint32_t dst = base + (j % stages) * L.stage + lane * 16;
#pragma unroll
    for (int i = 0; i < BK / NW; ++i) {
      const char* k = kbase + static_cast<size_t>(row0 + i * NW) * (wk * 2);
      const char* v = vbase + static_cast<size_t>(row0 + i * NW) * (wv * 2);
      const uint32_t dk_ = dst + (warp + i * NW) * L.pk * 2, dv_ = dst + L.off_v + (warp + i * NW) * L.pv * 2;
      for (int x = lane * 8, o = 0; x < wk; x += 256, o += 512) cp16(dk_ + o, k + o, true);
      for (int x = lane * 8, o = 0; x < wv; x += 256, o += 512) cp16(dv_ + o, v + o, true);
    }
    poff += BK;
    if (poff == a.page) {
      poff = 0;
      ++pidx;
      if (j + 1 < nt) pg = table[pidx];
    }
  };
  for (int j = 0; j < max(1, stages - 1); ++j) {
    if (j < nt) load(j);
    cp_commit();
  }
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + b * a.q_stride;
  for (int e = tid; e < (H + 1) * (L.pq / 8); e += NT) {
    const int r = e / (L.pq / 8), x = (e % (L.pq / 8)) * 8;
    *reinterpret_cast<uint4*>(sQ + r * L.pq + x) = r < H && x < dk ? *reinterpret_cast<const uint4*>(q + r * dk + x) : make_uint4(0u, 0u, 0u, 0u);
  }
  for (int e = tid; e < H * NW * HPW; e += NT) {  // target head of (warp, i): warp + NW i
    const int g = e / (NW * HPW), w = (e / HPW) % NW, h = w + NW * (e % HPW);
    sM[e] = h < H ? a.mix[h * H + g] * a.scale : 0.f;
  }
  for (int e = tid; e < PP; e += NT) sP[H * PP + e] = f2bf(0.f);
  if (tid == 0) sA[H] = 1.f;
  // columns behind a key row meet zero queries: they must be finite
  for (int e = tid; e < stages * BK; e += NT)
    *reinterpret_cast<uint4*>(msm + (e / BK) * L.stage + ((e % BK) * L.pk + wk) * 2) = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();

  float m_run[HPW], l_run[HPW];  // softmax state of heads warp, warp + NW, ..; the sum is a part per lane
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
  }
  float o[NB][2][4];
  int hab[NB], vcol[NB];  // per value block: heads of rows gq and gq + 8 of the operand (low, high half; H: none), first column
  uint32_t pa[NB];               // its weights: this lane's row
  const int dvb = (dv + 15) / 16, groups = a.KV * MT, blocks = groups * dvb;
#pragma unroll
  for (int i = 0; i < NB; ++i) {
    const int blk = warp + NW * i, m = blk / dvb, kvh = m / MT, h0 = (m % MT) * 16;
    auto head = [&](int r) { return blk < blocks && h0 + r < per ? kvh * per + h0 + r : H; };
    hab[i] = head(gq) | head(gq + 8) << 16;
    pa[i] = smem_u32(sP + head(lane & 15) * PP + (lane >> 4) * 8);
    vcol[i] = blk < blocks ? kvh * dv + (blk % dvb) * 16 : -1;
#pragma unroll
    for (int n = 0; n < 2; ++n) o[i][n][0] = o[i][n][1] = o[i][n][2] = o[i][n][3] = 0.f;
  }
  const int nks = (dk + 15) / 16;
  // raw scores: task i of this warp takes keys 8 kb .. of group m = warp / 4 + NW / 4 i (KV head m / MT, query heads 16 (m % MT) ..)
  const int kb = warp & 3, key_c = kb * 8 + 2 * t4;
  auto group_head = [&](int m, int r) { return (m % MT) * 16 + r < per ? (m / MT) * per + (m % MT) * 16 + r : H; };
  const uint32_t k_row = ((kb * 8 + (lane & 7)) * L.pk + (lane >> 3) * 8) * 2;
  uint32_t qr[NTK > 0 ? NTK : 1][NQ > 0 ? NQ : 1][4];
  uint32_t kofs[NTK > 0 ? NTK : 1];
  int sa[NTK > 0 ? NTK : 1], sb[NTK > 0 ? NTK : 1];  // where the scores go (negative: no such head)
  if constexpr (NTK > 0) {
#pragma unroll
    for (int i = 0; i < NTK; ++i) {
      const int m = (warp >> 2) + NW / 4 * i;
      const bool ok = m < groups;
      const int ra = ok ? group_head(m, gq) : H, rb = ok ? group_head(m, gq + 8) : H;
      sa[i] = ra < H ? ra * PS + key_c : -1;
      sb[i] = rb < H ? rb * PS + key_c : -1;
      kofs[i] = k_row + (ok ? m / MT : 0) * dk * 2;
      const uint32_t qa = smem_u32(sQ + (ok ? group_head(m, lane & 15) : H) * L.pq + (lane >> 4) * 8);
#pragma unroll
      for (int k = 0; k < NQ; ++k)
        if (k < nks) ldm_x4(qa + k * 32, qr[i][k]);
        else qr[i][k][0] = qr[i][k][1] = qr[i][k][2] = qr[i][k][3] = 0u;
    }
  }
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
    if constexpr (NTK > 0) {
      float s[NTK][2][4];
#pragma unroll
      for (int i = 0; i < NTK; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][0][e] = s[i][1][e] = 0.f;
#pragma unroll
      for (int k = 0; k < NQ; k += 2) {
        if (k + 1 < nks) {  // uniform
#pragma unroll
          for (int i = 0; i < NTK; ++i) {
            uint32_t kf[4];
            ldm_x4(st + kofs[i] + k * 32, kf);
            mma16816(s[i][0], qr[i][k], kf[0], kf[1]);
            mma16816(s[i][1], qr[i][k + 1], kf[2], kf[3]);
          }
        } else if (k < nks) {  // one step: lanes 16.. repeat the addresses of lanes 0..
#pragma unroll
          for (int i = 0; i < NTK; ++i) {
            uint32_t kf[4];
            ldm_x4(st + kofs[i] + k * 32 - ((lane >> 4) << 5), kf);
            mma16816(s[i][0], qr[i][k], kf[0], kf[1]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < NTK; ++i) {
        if (sa[i] >= 0) {
          sS[sa[i]] = s[i][0][0] + s[i][1][0];
          sS[sa[i] + 1] = s[i][0][1] + s[i][1][1];
        }
        if (sb[i] >= 0) {
          sS[sb[i]] = s[i][0][2] + s[i][1][2];
          sS[sb[i] + 1] = s[i][0][3] + s[i][1][3];
        }
      }
    } else {
      for (int m = warp >> 2; m < groups; m += NW / 4) {
        const uint32_t qa = smem_u32(sQ + group_head(m, lane & 15) * L.pq + (lane >> 4) * 8), ka = st + k_row + (m / MT) * dk * 2;
        float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
        int k = 0;
        for (; k + 1 < nks; k += 2) {
          uint32_t a0[4], a1[4], kf[4];
          ldm_x4(ka + k * 32, kf);
          ldm_x4(qa + k * 32, a0);
          ldm_x4(qa + k * 32 + 32, a1);
          mma16816(s0, a0, kf[0], kf[1]);
          mma16816(s1, a1, kf[2], kf[3]);
        }
        if (k < nks) {
          uint32_t a0[4], kf[4];
          ldm_x4(ka + k * 32 - ((lane >> 4) << 5), kf);
          ldm_x4(qa + k * 32, a0);
          mma16816(s0, a0, kf[0], kf[1]);
        }
        const int ra = group_head(m, gq), rb = group_head(m, gq + 8);
        if (ra < H) {
          sS[ra * PS + key_c] = s0[0] + s1[0];
          sS[ra * PS + key_c + 1] = s0[1] + s1[1];
        }
        if (rb < H) {
          sS[rb * PS + key_c] = s0[2] + s1[2];
          sS[rb * PS + key_c + 1] = s0[3] + s1[3];
        }
      }
    }
    __syncthreads();
    // ---- mixing and online softmax. The running maximum follows only when a score has outgrown it by more than 8.
    const int key = (t0 + it) * BK + lane;
    const bool visible = key < ctx && key >= first_key;
    bool grown = false;
    float v[HPW];
#pragma unroll
    for (int i = 0; i < HPW; ++i) v[i] = 0.f;
    {
      const float* mw = sM + warp * HPW;
      const float* sl = sS + lane;
#pragma unroll 8
      for (int g = 0; g < H; ++g) {
        const float x = sl[g * PS];
        if constexpr (HPW % 4 == 0) {
#pragma unroll
          for (int i = 0; i < HPW; i += 4) {
            const float4 w = *reinterpret_cast<const float4*>(mw + g * (NW * HPW) + i);
            v[i] += w.x * x;
            v[i + 1] += w.y * x;
            v[i + 2] += w.z * x;
            v[i + 3] += w.w * x;
          }
        } else {
          const float2 w = *reinterpret_cast<const float2*>(mw + g * (NW * HPW));
          v[0] += w.x * x;
          v[1] += w.y * x;
        }
      }
    }
#pragma unroll
    for (int i = 0; i < HPW; ++i) {
      const int h = warp + NW * i;
      if (h < H) {  // warp-uniform
        if (!visible) v[i] = -INFINITY;
        float alpha = 1.f;
        if (__any_sync(0xffffffffu, v[i] > m_run[i] + 8.f)) {
          const float mx = fmaxf(m_run[i], warp_max(v[i]));
          alpha = __expf(m_run[i] - mx);  // (exp of -infinity: 0)
          m_run[i] = mx;
          l_run[i] *= alpha;
          grown = true;
        }
        const float p = v[i] == -INFINITY ? 0.f : __expf(v[i] - m_run[i]);
        l_run[i] += p;
        sP[h * PP + lane] = f2bf(p);
        if (lane == 0) sA[h] = alpha;
      }
    }
    const bool rescale = __syncthreads_or(grown);
    // ---- weighted sums: warp w owns the 16-column blocks w, w + NW, ..
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      if (vcol[i] < 0) continue;  // warp-uniform
      if (rescale) {
        const float fa = sA[hab[i] & 0xffff], fb = sA[hab[i] >> 16];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          o[i][n][0] *= fa;
          o[i][n][1] *= fa;
          o[i][n][2] *= fb;
          o[i][n][3] *= fb;
        }
      }
      const uint32_t va = st + L.off_v + (((lane & 7) + ((lane >> 3) & 1) * 8) * L.pv + vcol[i] + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int ks = 0; ks < BK / 16; ++ks) {
        uint32_t p4[4], v4[4];
        ldm_x4(pa[i] + ks * 32, p4);
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
    const int h = warp + NW * i;
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
      const int h = half ? hab[i] >> 16 : hab[i] & 0xffff;
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

template <int NW, int HPW, int NB, int NTK, int NQ>
static int launch_mixed_decode_t(const MixedDecodeArgs& a, const MixedPlan& p, cudaStream_t st) {
  static PerDeviceOnce once;
  if (once.first() && cudaFuncSetAttribute(mixed_decode_kernel<NW, HPW, NB, NTK, NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return 2;
  const size_t smem = static_cast<size_t>(MixedDecodeSmem(a.H, a.KV, a.dk, a.dv, p.stages, NW * HPW).bytes);
  if (launch_pdl(mixed_decode_kernel<NW, HPW, NB, NTK, NQ>, dim3(a.splits, a.B), dim3(NW * 32), smem, st, a, p.stages) != cudaSuccess) return 2;
  if (a.splits > 1) launch_decode_merge(a.part_o, a.part_ml, a.out, a.B, a.H, a.dv, a.splits, a.x, st);
  return 0;
}

int launch_mixed_decode(const MixedDecodeArgs& a, cudaStream_t st) {
  if (a.B == 0) return 0;
  const MixedPlan p = mixed_plan(a.H, a.KV, a.dk, a.dv);
  if (p.warps == 0 || a.page % kMxBK != 0 || a.q_stride % 8 != 0 || a.B > 65535 || a.splits < 1 || a.x.sink != nullptr || (a.x.gate != nullptr && !a.x.gate_heads)) return 1;
#define DLV_MIXED(W, HP, NBV, TK, Q) \
  if (p.warps == W && p.hpw == HP && p.blocks == NBV && p.tasks == TK && p.steps == Q) return launch_mixed_decode_t<W, HP, NBV, TK, Q>(a, p, st)
#define DLV_MIXED4(W, TK, Q)  \
  DLV_MIXED(W, 2, 2, TK, Q);  \
  DLV_MIXED(W, 2, 4, TK, Q);  \
  DLV_MIXED(W, 4, 2, TK, Q);  \
  DLV_MIXED(W, 4, 4, TK, Q)
  DLV_MIXED4(8, 2, 4);
  DLV_MIXED4(8, 1, 8);
  DLV_MIXED4(16, 1, 8);
  DLV_MIXED4(16, 2, 8);
  DLV_MIXED(8, 8, 2, 0, 0);
  DLV_MIXED(8, 8, 4, 0, 0);
  DLV_MIXED(8, 8, 8, 0, 0);
#undef DLV_MIXED4
#undef DLV_MIXED
  return 1;
}

// out [T, H, pitch >= KV dk]. A thread takes eight columns of one (row, KV head): the group's queries stay in registers (PER > 0 of them) while it goes over the
// heads; PER = 0: groups of any size, read again for every head.
template <typename TIO, int PER>
__global__ void __launch_bounds__(256) fold_heads_kernel(const TIO* __restrict__ q, long long q_stride, const float* __restrict__ mix, TIO* __restrict__ out,
                                                         int pitch, int H, int KV, int dk, int rows) {
  extern __shared__ float fsm[];  // [H][H]
  pdl_wait();
  pdl_trigger();
  for (int e = threadIdx.x; e < H * H; e += 256) fsm[e] = mix[e];
  __syncthreads();
  const int vecs = dk / 8, per = PER > 0 ? PER : H / KV, n = rows * KV * vecs;
  const int idx = blockIdx.x * 256 + threadIdx.x;
  if (idx >= n) return;
  const int x = (idx % vecs) * 8, kvh = (idx / vecs) % KV, t = idx / (vecs * KV);
  const TIO* src = q + t * q_stride + static_cast<long long>(kvh * per) * dk + x;
  float v[PER > 0 ? PER : 1][8];
  if constexpr (PER > 0) {
#pragma unroll
    for (int g = 0; g < PER; ++g) io_ld8(src + g * dk, v[g]);
  }
  TIO* dst = out + static_cast<long long>(t) * H * pitch + kvh * dk + x;
  const float* m = fsm + kvh * per;
#pragma unroll 2
  for (int h = 0; h < H; ++h) {
    float acc[8] = {};
    if constexpr (PER > 0) {
#pragma unroll
      for (int g = 0; g < PER; ++g) {
        const float w = m[g];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] += w * v[g][e];
      }
    } else {
      for (int g = 0; g < per; ++g) {
        io_ld8(src + g * dk, v[0]);
        const float w = m[g];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] += w * v[0][e];
      }
    }
    io_st8(dst, acc);
    dst += pitch;
    m += H;
  }
}

template <typename TIO>
static void launch_fold_heads_t(const void* q, long long q_stride, const float* mix, void* out, int pitch, int T, int H, int KV, int dk, cudaStream_t st) {
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(T) * KV * (dk / 8) + 255) / 256));
  const size_t smem = static_cast<size_t>(H) * H * 4;
#define DLV_FOLD(N) launch_pdl(fold_heads_kernel<TIO, N>, grid, dim3(256), smem, st, static_cast<const TIO*>(q), q_stride, mix, static_cast<TIO*>(out), pitch, H, KV, dk, T)
  switch (H / KV) {
    case 1: DLV_FOLD(1); break;
    case 2: DLV_FOLD(2); break;
    case 3: DLV_FOLD(3); break;
    case 4: DLV_FOLD(4); break;
    case 5: DLV_FOLD(5); break;
    case 6: DLV_FOLD(6); break;
    case 8: DLV_FOLD(8); break;
    default: DLV_FOLD(0);
  }
#undef DLV_FOLD
}
int launch_fold_heads(const void* q, long long q_stride, const float* mix, void* out, int pitch, int T, int H, int KV, int dk, bool is_f32, cudaStream_t st) {
  if (T == 0) return 0;
  if (H > 108 || static_cast<long long>(T) * KV * (dk / 8) > 0x7fffff00ll) return 1;  // (the matrix fits 48 KB of shared memory)
  if (is_f32) launch_fold_heads_t<float>(q, q_stride, mix, out, pitch, T, H, KV, dk, st);
  else launch_fold_heads_t<__nv_bfloat16>(q, q_stride, mix, out, pitch, T, H, KV, dk, st);
  return 0;
}

}  // namespace dlv
