// Prompt attention of the layer-stack decoder on the tensor pipe: sliding window with the first tokens
// kept, grouped heads, bf16 queries / keys / values, f32 scores, weights and accumulation, with the
// sigmoid output gate in the epilogue.  A key is a row of its head, or that and a part that all heads
// share (the expanded keys and the rotated part of a latent attention).
//
// One CTA = 64 query rows of one head (4 warps of 16 rows) walking the keys its rows can see: the kept
// positions first, then the window of its first row up to its last row, 64 keys a tile, fetched row by
// row from the cache's kept slots and ring with 16-byte cp.async into a double buffer.  Scores and
// products are mma.sync m16n8k16 with bf16 operands; a tile that every row of a warp sees whole skips
// the mask.  Query/key widths up to 192, values up to 128 (rounded up to a tile width with zero columns).
#include "mixers.cuh"
#include "rows_mma.cuh"

namespace tlb {

namespace {

constexpr int AW_M = 64, AW_N = 64, AW_THREADS = 128;

__device__ __forceinline__ uint32_t aw_pack(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *(const uint32_t*)&h;
}

template <int DK, int DV>
struct AwSmem {
  static constexpr int LK = DK + 8, LV = DV + 8;          // row strides in elements
  static constexpr size_t Q = 0;
  static constexpr size_t K = Q + (size_t)AW_M * LK * 2;
  static constexpr size_t V = K + (size_t)2 * AW_N * LK * 2;
  static constexpr size_t TOTAL = V + (size_t)2 * AW_N * LV * 2;
};

__device__ __forceinline__ int aw_slot(const AttnTiles& p, int j) {
  return j < p.keep ? j : p.keep + (int)((unsigned)(j - p.keep) % (unsigned)p.ring);
}

template <int DK, int DV>
__global__ void __launch_bounds__(AW_THREADS, 2)
    attn_window_kernel(const __grid_constant__ AttnTiles p, __nv_bfloat16* __restrict__ out, long long ldo, int rows,
                       int pos0) {
  using S = AwSmem<DK, DV>;
  using B = __nv_bfloat16;
  constexpr int LK = S::LK, LV = S::LV, CK = DK / 8, CV = DV / 8;
  extern __shared__ __align__(16) unsigned char smem[];
  B* qs = (B*)(smem + S::Q);
  B* ks = (B*)(smem + S::K);
  B* vs = (B*)(smem + S::V);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = (gridDim.x - 1 - blockIdx.x) * AW_M, h = blockIdx.y, g = h / p.R;
  const int nrow = rows - r0 < AW_M ? rows - r0 : AW_M;
  const int dch = p.kw / 8, qch = dch + p.k2w / 8, ech = p.vw / 8;
  // zero columns behind the widths: never written again
  for (int i = tid; i < (int)(S::TOTAL / 16); i += AW_THREADS) ((uint4*)smem)[i] = make_uint4(0, 0, 0, 0);
  pdl_wait();
  pdl_launch_dependents();
  __syncthreads();
  for (int i = tid; i < nrow * qch; i += AW_THREADS) {
    const int r = i / qch, c = i - r * qch;
    rc_cp16(qs + r * LK + c * 8, (const B*)p.q + (size_t)(r0 + r) * p.q_row + h * p.q_head + c * 8, true);
  }
  // what the block's rows can see: kept positions in front of the first row's window, then the window
  const int pf = pos0 + r0, pl = pf + nrow - 1;
  Visible vis;
  vis.lo = pf + 1 > p.window ? pf + 1 - p.window : 0;
  vis.kept = p.keep < vis.lo ? p.keep : vis.lo;
  vis.n = vis.kept + pl + 1 - vis.lo;
  const B *K = (const B*)p.k + (size_t)g * p.k_head, *K2 = (const B*)p.k2, *V = (const B*)p.v + (size_t)g * p.v_head;
  auto fetch = [&](int tile, int buf) {
    // two threads a key row, one half of its chunks each
    const int r = tid >> 1, half = tid & 1, t = tile * AW_N + r;
    const bool on = t < vis.n;
    const size_t slot = aw_slot(p, on ? visible_pos(vis, t) : pl);
    const B *kr = K + slot * p.k_row, *kr2 = K2 + slot * p.k2_row - dch * 8, *vr = V + slot * p.v_row;
    B *kd = ks + (buf * AW_N + r) * LK, *vd = vs + (buf * AW_N + r) * LV;
#pragma unroll
    for (int i = 0; i < CK / 2; i++) {
      const int c = 2 * i + half;
      if (c < dch) rc_cp16(kd + c * 8, kr + c * 8, on);
      else if (c < qch) rc_cp16(kd + c * 8, kr2 + c * 8, on);
    }
#pragma unroll
    for (int i = 0; i < CV / 2; i++) {
      const int c = 2 * i + half;
      if (c < ech) rc_cp16(vd + c * 8, vr + c * 8, on);
    }
  };
  const int ntile = (vis.n + AW_N - 1) / AW_N;
  fetch(0, 0);
  rc_commit();
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-1.0e30f, -1.0e30f}, l[2] = {0.f, 0.f};
  uint32_t qf[DK / 16][4];
  const int wr = warp * 16, row_a = wr + (lane >> 2), col_a = (lane & 3) * 2;
  const int pa = pf + row_a, pb = pa + 8;                 // positions of the thread's two rows
  const int wp0 = pf + wr, wp1 = wp0 + 15;                // of the warp's
  const float sl2 = p.scale * 1.4426950408889634f;
  for (int t = 0; t < ntile; t++) {
    const int buf = t & 1;
    if (t + 1 < ntile) {
      fetch(t + 1, buf ^ 1);
      rc_commit();
      rc_wait<1>();
    } else {
      rc_wait<0>();
    }
    __syncthreads();
    if (t == 0) {
#pragma unroll
      for (int k = 0; k < DK / 16; k++)
        rc_ldm(qf[k], qs + (wr + (lane & 15)) * LK + k * 16 + (lane >> 4) * 8);
    }
    const int i0 = t * AW_N, i1 = (i0 + AW_N < vis.n ? i0 + AW_N : vis.n) - 1;
    const int j0 = visible_pos(vis, i0), j1 = visible_pos(vis, i1);
    // positions of a tile increase with the index, so its ends tell whether the warp sees all / nothing of it
    const bool none = j0 > wp1 || (wp0 - j1 >= p.window && j0 >= p.keep);
    if (!none) {
      const bool whole = i1 - i0 == AW_N - 1 && j1 <= wp0 && (wp1 - j0 < p.window || j1 < p.keep);
      float s[8][4];
#pragma unroll
      for (int n = 0; n < 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const B* kb = ks + buf * AW_N * LK;
#pragma unroll
      for (int k = 0; k < DK / 16; k++)
#pragma unroll
        for (int n = 0; n < 4; n++) {
          uint32_t b[4];
          rc_ldm(b, kb + (n * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + k * 16 + ((lane >> 3) & 1) * 8);
          rc_mma(s[2 * n], qf[k], b[0], b[1]);
          rc_mma(s[2 * n + 1], qf[k], b[2], b[3]);
        }
      if (!whole) {
#pragma unroll
        for (int n = 0; n < 8; n++)
#pragma unroll
          for (int e = 0; e < 4; e++) {
            const int i = i0 + n * 8 + col_a + (e & 1), j = visible_pos(vis, i), pp = e < 2 ? pa : pb;
            if (i > i1 || j > pp || (pp - j >= p.window && j >= p.keep)) s[n][e] = -INFINITY;
          }
      }
      float mx[2] = {m[0], m[1]};
#pragma unroll
      for (int n = 0; n < 8; n++) {
        mx[0] = fmaxf(mx[0], fmaxf(s[n][0], s[n][1]) * sl2);
        mx[1] = fmaxf(mx[1], fmaxf(s[n][2], s[n][3]) * sl2);
      }
#pragma unroll
      for (int e = 0; e < 2; e++) {
        mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
        mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
        const float c = exp2f(m[e] - mx[e]);
        m[e] = mx[e];
        l[e] *= c;
#pragma unroll
        for (int i = 0; i < DV / 8; i++) { o[i][2 * e] *= c; o[i][2 * e + 1] *= c; }
      }
      uint32_t pf_[4][4];
#pragma unroll
      for (int n = 0; n < 8; n++) {
        float w[4];
#pragma unroll
        for (int e = 0; e < 4; e++) w[e] = exp2f(fmaf(s[n][e], sl2, -m[e >> 1]));
        l[0] += w[0] + w[1];
        l[1] += w[2] + w[3];
        pf_[n >> 1][(n & 1) * 2] = aw_pack(w[0], w[1]);
        pf_[n >> 1][(n & 1) * 2 + 1] = aw_pack(w[2], w[3]);
      }
      const B* vb = vs + buf * AW_N * LV;
#pragma unroll
      for (int k = 0; k < 4; k++)
#pragma unroll
        for (int n = 0; n < DV / 16; n++) {
          uint32_t b[4];
          rc_ldmt(b, vb + (k * 16 + (lane & 15)) * LV + n * 16 + (lane >> 4) * 8);
          rc_mma(o[2 * n], pf_[k], b[0], b[1]);
          rc_mma(o[2 * n + 1], pf_[k], b[2], b[3]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int e = 0; e < 2; e++) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
    const int r = row_a + 8 * e;
    if (r >= nrow) continue;
    const float inv = p.out_scale / l[e];
    const float* gate = p.gate ? p.gate + (size_t)(r0 + r) * p.gate_row + h * p.E : nullptr;
    B* dst = out + (size_t)(r0 + r) * ldo + h * p.E;
#pragma unroll
    for (int n = 0; n < DV / 8; n++) {
      const int c = n * 8 + col_a;
      float a = o[n][2 * e] * inv, b = o[n][2 * e + 1] * inv;
      if ((p.E & 1) == 0) {
        if (c < p.E) {
          if (gate) {
            const float2 gt = *(const float2*)(gate + c);
            a *= sigmoid_f(gt.x);
            b *= sigmoid_f(gt.y);
          }
          *(uint32_t*)(dst + c) = aw_pack(a, b);
        }
      } else {
        if (c < p.E) dst[c] = __float2bfloat16_rn(gate ? a * sigmoid_f(gate[c]) : a);
        if (c + 1 < p.E) dst[c + 1] = __float2bfloat16_rn(gate ? b * sigmoid_f(gate[c + 1]) : b);
      }
    }
  }
}

template <int DK, int DV>
int aw_launch(const AttnTiles& p, void* out, long long ldo, int rows, int pos0, cudaStream_t s) {
  constexpr int smem = (int)AwSmem<DK, DV>::TOTAL;
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(attn_window_kernel<DK, DV>, smem, done);
  if (rc) return rc;
  LaunchCfg lc(dim3((rows + AW_M - 1) / AW_M, p.H), dim3(AW_THREADS), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, attn_window_kernel<DK, DV>, p, (__nv_bfloat16*)out, ldo, rows, pos0));
  return TLB_OK;
}

}  // namespace

bool attn_tiles_eligible(int qk_width, int v_width) { return qk_width <= 192 && v_width <= 128; }

int attn_tiles_launch(const AttnTiles& t, void* out, long long ldo, int rows, int pos0, cudaStream_t s) {
  const int k = t.kw + t.k2w, v = t.vw, w = k > v ? k : v;
  if (!attn_tiles_eligible(k, v)) return set_error(TLB_ERR_UNSUPPORTED, "attention tiles: head too wide");
  if (w <= 32) return aw_launch<32, 32>(t, out, ldo, rows, pos0, s);
  if (w <= 64) return aw_launch<64, 64>(t, out, ldo, rows, pos0, s);
  if (w <= 96) return aw_launch<96, 96>(t, out, ldo, rows, pos0, s);
  if (w <= 128) return aw_launch<128, 128>(t, out, ldo, rows, pos0, s);
  return aw_launch<192, 128>(t, out, ldo, rows, pos0, s);
}

bool attn_window_eligible(const AttnP& p) { return p.Dp <= 128 && p.Ep <= 128; }

int attn_window_launch(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda,
                       int rows, int pos0, cudaStream_t s) {
  AttnTiles t{};
  t.q = q; t.q_row = (long long)p.H * p.Dp; t.q_head = p.Dp;
  t.k = p.K; t.k_row = p.Dp; t.k_head = (long long)p.cap * p.Dp; t.kw = p.Dp;
  t.v = p.V; t.v_row = p.Ep; t.v_head = (long long)p.cap * p.Ep; t.vw = p.Ep;
  t.H = p.H; t.R = p.H / p.G; t.E = p.E;
  t.window = p.window; t.keep = p.keep; t.ring = p.ring;
  t.scale = p.scale; t.out_scale = p.out_scale;
  t.gate = proj + p.og; t.gate_row = ld;
  return attn_tiles_launch(t, (__nv_bfloat16*)act + p.oa, lda, rows, pos0, s);
}

}  // namespace tlb
