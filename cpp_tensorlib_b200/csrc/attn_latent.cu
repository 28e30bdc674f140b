// Latent attention of the layer-stack decoder.  What a position keeps is one row for all heads: the
// normed latent c [C] and the rotated key part r [R].  With the rows of W_uk and W_uv of a head,
//   score = (q_n . W_uk c + q_r . r) scale = (W_uk^T q_n . c + q_r . r) scale,   value = W_uv c,
// so a query is taken to the latent's side once (absorb), the attention runs on the kept rows as one
// key/value head of width C + R that every head shares (attend), and the weighted latent goes through
// W_uv once (fold, with the output gate).  A token and short runs of rows take this form; in bf16 the
// attention is mma.sync m16n8k16 with 16 heads as the rows of a tile.  Long prompt passes in bf16 expand
// keys and values of the visible rows instead and run on the tiles of attn_window.cu.
//
// Key ranges of a position are independent blocks; the fold merges them.
#include "mixers.cuh"
#include "rows_mma.cuh"

namespace tlb {

namespace {

constexpr int LA_THREADS = 256, LA_COLS = 64, LA_EROWS = 16;

// kept rows that `pos` sees, cut into ranges of a multiple of 64
struct LatentRange { int lo, n, chunk, active; };
__device__ __forceinline__ LatentRange latent_range(const LatentP& p, int pos, int splits) {
  LatentRange r;
  r.lo = pos + 1 > p.window ? pos + 1 - p.window : 0;
  r.n = pos + 1 - r.lo;
  r.chunk = ((r.n + splits - 1) / splits + 63) & ~63;
  r.active = (r.n + r.chunk - 1) / r.chunk;
  return r;
}
__device__ __forceinline__ int latent_slot(const LatentP& p, int j) { return (int)((unsigned)j % (unsigned)p.ring); }
__device__ __forceinline__ int pos_of(const unsigned* d_pos, int pos0, int row) { return d_pos ? (int)*d_pos : pos0 + row; }

// element r of a rotated row of R elements at `src`
__device__ __forceinline__ float rot_pair(const LatentP& p, const float* src, const float2* cs, int r) {
  if (r >= p.R) return 0.f;
  const int e = r & ~1;
  const float u = src[e], v = src[e + 1];
  const float2 t = cs[r >> 1];
  return (r & 1) ? v * t.x + u * t.y : u * t.x - v * t.y;
}
__device__ __forceinline__ void rot_row_table(const LatentP& p, int pos, float2* cs) {
  for (int i = threadIdx.x; i < p.R / 2; i += blockDim.x) rot_angle(pos, p.inv_freq[i], &cs[i].y, &cs[i].x);
}
// the kept row of one position from its projected row; the whole block, cs filled, barriers inside
template <typename KT>
__device__ void latent_keep(const LatentP& p, const float* row, int pos, const float2* cs, float* red) {
  float sq = 0.f;
  for (int i = threadIdx.x; i < p.C; i += blockDim.x) { const float v = row[p.oc + i]; sq = fmaf(v, v, sq); }
  const float r = rsqrtf(block_sum(sq, red) / p.C + p.eps);
  KT* dst = (KT*)p.rows + (size_t)latent_slot(p, pos) * p.row();
  for (int i = threadIdx.x; i < p.Cp; i += blockDim.x) put(dst + i, i < p.C ? row[p.oc + i] * r * p.cn[i] : 0.f);
  for (int i = threadIdx.x; i < p.Rp; i += blockDim.x) put(dst + p.Cp + i, rot_pair(p, row + p.oc + p.Cp, cs, i));
}

// ---- prompt pass: normed query latents, kept rows ---------------------------------------------
template <typename KT>
__global__ void __launch_bounds__(LA_THREADS) latent_prep_kernel(const __grid_constant__ LatentP p,
                                                                 const float* __restrict__ proj, long long ld, int pos0,
                                                                 KT* __restrict__ qlat) {
  __shared__ float red[33];
  __shared__ float2 cs[MX_PAIRS];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, pos = pos0 + t;
  const float* row = proj + (size_t)t * ld;
  if (p.owner) rot_row_table(p, pos, cs);
  float sq = 0.f;
  for (int i = threadIdx.x; i < p.Q; i += LA_THREADS) { const float v = row[p.oq + i]; sq = fmaf(v, v, sq); }
  const float r = rsqrtf(block_sum(sq, red) / p.Q + p.eps);
  for (int i = threadIdx.x; i < p.Qp; i += LA_THREADS)
    put(qlat + (size_t)t * p.Qp + i, i < p.Q ? row[p.oq + i] * r * p.qn[i] : 0.f);
  if (p.owner) latent_keep<KT>(p, row, pos, cs, red);
}

// ---- queries to the latent's side -------------------------------------------------------------
// Block (64 latent columns, head, row): a thread owns 16 bytes of the columns and every DG-th query
// dimension, whose weights it fetches before the queries are there.  The block behind the last column
// slice of head 0 keeps the token's own row.
constexpr int LB_PRE = 4;
template <typename KT>
__global__ void __launch_bounds__(LA_THREADS) latent_absorb_kernel(const __grid_constant__ LatentP p,
                                                                   const float* __restrict__ q, long long ldq,
                                                                   const float* __restrict__ proj, KT* __restrict__ qa,
                                                                   const unsigned* d_pos, int pos0) {
  constexpr int CE = Vec16<KT>::N, CH = LA_COLS / CE, DG = LA_THREADS / CH;
  __shared__ float2 cs[MX_PAIRS];
  __shared__ float part[DG][LA_COLS + 1];
  __shared__ float red[33];
  __shared__ float qs[1024];
  const int tid = threadIdx.x, h = blockIdx.y, row = blockIdx.z, c0 = blockIdx.x * LA_COLS;
  const int pos = pos_of(d_pos, pos0, row);
  if (c0 >= p.Cp) {   // the kept row (one token only)
    rot_row_table(p, pos, cs);
    pdl_wait();
    pdl_launch_dependents();
    if (h == 0) latent_keep<KT>(p, proj, pos, cs, red);
    return;
  }
  const int ch = tid % CH, dg = tid / CH, c = c0 + ch * CE;
  const KT* W = (const KT*)p.ukv + (size_t)h * p.Dp * p.Cp + c;
  const bool on = c < p.Cp;
  uint4 w[LB_PRE];
#pragma unroll
  for (int i = 0; i < LB_PRE; i++) {
    const int d = dg + i * DG;
    w[i] = on && d < p.D ? *(const uint4*)(W + (size_t)d * p.Cp) : make_uint4(0, 0, 0, 0);
  }
  if (blockIdx.x == 0) rot_row_table(p, pos, cs);
  pdl_wait();
  pdl_launch_dependents();
  const float* src = q + (size_t)row * ldq + (size_t)h * p.qw();
  for (int d = tid; d < p.D; d += LA_THREADS) qs[d] = src[d];
  __syncthreads();
  float acc[CE];
#pragma unroll
  for (int e = 0; e < CE; e++) acc[e] = 0.f;
  for (int d0 = 0; d0 < p.D; d0 += LB_PRE * DG) {
    if (d0) {
#pragma unroll
      for (int i = 0; i < LB_PRE; i++) {
        const int d = d0 + dg + i * DG;
        w[i] = on && d < p.D ? *(const uint4*)(W + (size_t)d * p.Cp) : make_uint4(0, 0, 0, 0);
      }
    }
#pragma unroll
    for (int i = 0; i < LB_PRE; i++) {
      const int d = d0 + dg + i * DG;
      if (d < p.D) {
        float f[CE];
        widen16(w[i], f, (const KT*)nullptr);
        const float x = qs[d];
#pragma unroll
        for (int e = 0; e < CE; e++) acc[e] = fmaf(f[e], x, acc[e]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < CE; e++) part[dg][ch * CE + e] = acc[e];
  __syncthreads();
  KT* dst = qa + ((size_t)row * p.H + h) * p.row();
  // four threads a column, then their sums
  const int col = tid >> 2, quarter = tid & 3;
  float s = 0.f;
  for (int i = quarter; i < DG; i += 4) s += part[i][col];
  s += __shfl_xor_sync(0xffffffffu, s, 1);
  s += __shfl_xor_sync(0xffffffffu, s, 2);
  if (quarter == 0 && c0 + col < p.Cp) put(dst + c0 + col, s);
  if (blockIdx.x == 0)
    for (int r = tid; r < p.Rp; r += LA_THREADS) put(dst + p.Cp + r, rot_pair(p, src + p.Dp, cs, r));
}

// ---- attention on the kept rows ----------------------------------------------------------------
// Partials: [row][range][H][Cp] unnormalised, then [row][range][H] (maximum, sum).
__device__ __forceinline__ float* part_of(const LatentP& p, float* part, int splits, int row, int split) {
  return part + ((size_t)row * splits + split) * p.H * p.Cp;
}
__device__ __forceinline__ const float* part_of(const LatentP& p, const float* part, int splits, int row, int split) {
  return part + ((size_t)row * splits + split) * p.H * p.Cp;
}
__device__ __forceinline__ float2* stat_of(const LatentP& p, float* part, int splits, int rows, int row, int split) {
  return (float2*)(part + (size_t)rows * splits * p.H * p.Cp) + ((size_t)row * splits + split) * p.H;
}

// any widths, either type: block (range, RM heads, row); 512 of the latent's columns at a time
constexpr int LA_VALUES = 2 * MX_THREADS;
template <typename KT, int RM>
__global__ void __launch_bounds__(LA_THREADS) latent_attend_kernel(const __grid_constant__ LatentP p,
                                                                   const KT* __restrict__ qa, float* __restrict__ part,
                                                                   int splits, const unsigned* d_pos, int pos0) {
  extern __shared__ __align__(16) float sm[];
  const int row = blockIdx.z, h0 = blockIdx.y * RM, tid = threadIdx.x, pos = pos_of(d_pos, pos0, row);
  const int nh = p.H - h0 < RM ? p.H - h0 : RM;
  const LatentRange lr = latent_range(p, pos, splits);
  pdl_wait();
  pdl_launch_dependents();
  if ((int)blockIdx.x >= lr.active) return;
  AttnP a{};
  a.Dp = p.row(); a.Vs = p.row(); a.cap = a.ring = p.ring; a.keep = 0; a.scale = p.scale;
  a.K = p.rows;
  float* qs = sm;
  float* os = qs + RM * a.Dp;
  float* sc = os + RM * (p.Cp < LA_VALUES ? p.Cp : LA_VALUES);
  float* ml = sc + RM * MX_TK;
  for (int i = tid; i < RM * a.Dp; i += LA_THREADS)
    qs[i] = i < nh * a.Dp ? to_f(qa[((size_t)row * p.H + h0) * a.Dp + i]) : 0.f;
  Visible vis;
  vis.kept = 0; vis.lo = lr.lo; vis.n = lr.n;
  const int t0 = blockIdx.x * lr.chunk, t1 = t0 + lr.chunk < lr.n ? t0 + lr.chunk : lr.n;
  float* dst = part_of(p, part, splits, row, blockIdx.x) + (size_t)h0 * p.Cp;
  for (int c0 = 0; c0 < p.Cp; c0 += LA_VALUES) {
    a.V = (KT*)p.rows + c0;
    a.Ep = p.Cp - c0 < LA_VALUES ? p.Cp - c0 : LA_VALUES;
    __syncthreads();
    attn_range<KT, RM>(a, qs, 0, vis, t0, t1, sc, os, ml);
    for (int i = tid; i < nh * a.Ep; i += LA_THREADS) {
      const int r = i / a.Ep;
      dst[(size_t)r * p.Cp + c0 + i - r * a.Ep] = os[i];
    }
  }
  if (tid < nh) stat_of(p, part, splits, gridDim.z, row, blockIdx.x)[h0 + tid] = make_float2(ml[tid], ml[RM + tid]);
}

// bf16: block (range, 16 heads, row), 64 kept rows a tile in a double buffer.  Scores: a warp takes 8 of
// the tile's keys; values: a warp takes 16 * NP of the latent's columns.  Weights enter the second product
// as two bf16 planes.
constexpr int LM_KEYS = 64, LM_PLD = LM_KEYS + 8;
struct LmSmem {
  int ld;                      // row stride in elements: the row rounded up to 16, plus 8
  size_t q, k, p, s, total;
  __host__ __device__ explicit LmSmem(int row) {
    ld = ((row + 15) & ~15) + 8;
    q = 0;
    k = q + (size_t)16 * ld * 2;
    p = k + (size_t)2 * LM_KEYS * ld * 2;
    s = p + (size_t)2 * 16 * LM_PLD * 2;
    total = s + (size_t)(16 * (LM_KEYS + 1) + 48) * 4;
  }
};
template <int NP>
__global__ void __launch_bounds__(LA_THREADS) latent_attend_mma_kernel(const __grid_constant__ LatentP p,
                                                                       const __nv_bfloat16* __restrict__ qa,
                                                                       float* __restrict__ part, int splits,
                                                                       const unsigned* d_pos, int pos0) {
  using B = __nv_bfloat16;
  extern __shared__ __align__(16) unsigned char smem[];
  const LmSmem L(p.row());
  B* qs = (B*)(smem + L.q);
  B* ks = (B*)(smem + L.k);
  B* ps = (B*)(smem + L.p);                // [2 planes][16][LM_PLD]
  float* ss = (float*)(smem + L.s);        // [16][65]
  float* corr = ss + 16 * (LM_KEYS + 1);   // [16]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row = blockIdx.z, h0 = blockIdx.y * 16;
  const int nh = p.H - h0 < 16 ? p.H - h0 : 16, ld = L.ld, rw = p.row(), ch = rw / 8, kst = (rw + 15) / 16;
  const int pos = pos_of(d_pos, pos0, row);
  const LatentRange lr = latent_range(p, pos, splits);
  if ((int)blockIdx.x >= lr.active) { pdl_wait(); pdl_launch_dependents(); return; }
  const int t0 = blockIdx.x * lr.chunk, t1 = t0 + lr.chunk < lr.n ? t0 + lr.chunk : lr.n;
  const int ntile = (t1 - t0 + LM_KEYS - 1) / LM_KEYS;
  auto fetch = [&](int tile, int buf) {   // four threads a row
    const int r = tid >> 2, t = t0 + tile * LM_KEYS + r;
    const bool on = t < t1;
    const B* src = (const B*)p.rows + (size_t)latent_slot(p, lr.lo + (on ? t : t0)) * rw;
    B* dst = ks + (buf * LM_KEYS + r) * ld;
#pragma unroll 6
    for (int c = tid & 3; c < ch; c += 4) rc_cp16(dst + c * 8, src + c * 8, on);
  };
  // columns that a product reads behind the row's own
  for (int i = tid; i < (16 + 2 * LM_KEYS) * (ld - rw) / 8; i += LA_THREADS) {
    const int r = i / ((ld - rw) / 8), c = i - r * ((ld - rw) / 8);
    *(uint4*)(qs + r * ld + rw + c * 8) = make_uint4(0, 0, 0, 0);
  }
  for (int i = tid; i < (16 - nh) * ch; i += LA_THREADS) {
    const int r = i / ch, c = i - r * ch;
    *(uint4*)(qs + (nh + r) * ld + c * 8) = make_uint4(0, 0, 0, 0);
  }
  // rows in front of the position itself were kept at least two launches ago
  const bool early = t0 + LM_KEYS < lr.n;
  if (early) fetch(0, 0);
  pdl_wait();
  pdl_launch_dependents();
  if (!early) fetch(0, 0);
  for (int i = tid; i < nh * ch; i += LA_THREADS) {
    const int r = i / ch, c = i - r * ch;
    rc_cp16(qs + r * ld + c * 8, qa + ((size_t)row * p.H + h0 + r) * rw + c * 8, true);
  }
  rc_commit();
  float o[2 * NP][4];
#pragma unroll
  for (int i = 0; i < 2 * NP; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int col0 = warp * 16 * NP, ra = lane >> 2, ca = (lane & 3) * 2;
  float m[2] = {-1.0e30f, -1.0e30f}, l[2] = {0.f, 0.f};   // of the warp's two heads: 2 warp, 2 warp + 1
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
    const B* kb = ks + buf * LM_KEYS * ld;
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    // four quarters of 32 dimensions' worth of 8 keys a load: two steps of 16
    const B* kr = kb + (warp * 8 + (lane & 7)) * ld + (lane >> 3) * 8;
    int k = 0;
#pragma unroll 4
    for (; k + 1 < kst; k += 2) {
      uint32_t a0[4], a1[4], b[4];
      rc_ldm(a0, rc_a(qs, ld, 0, k * 16, lane));
      rc_ldm(a1, rc_a(qs, ld, 0, k * 16 + 16, lane));
      rc_ldm(b, kr + k * 16);
      rc_mma(s0, a0, b[0], b[1]);
      rc_mma(s1, a1, b[2], b[3]);
    }
    if (k < kst) {   // the last 16: the upper half of the load repeats the lower
      uint32_t a0[4], b[4];
      rc_ldm(a0, rc_a(qs, ld, 0, k * 16, lane));
      rc_ldm(b, kb + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8 + k * 16);
      rc_mma(s0, a0, b[0], b[1]);
    }
    const int left = t1 - t0 - t * LM_KEYS;
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int key = warp * 8 + ca + (e & 1);
      ss[(ra + (e >> 1) * 8) * (LM_KEYS + 1) + key] = key < left ? (s0[e] + s1[e]) * sl2 : -INFINITY;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const int r = warp * 2 + j;
      const float x0 = ss[r * (LM_KEYS + 1) + 2 * lane], x1 = ss[r * (LM_KEYS + 1) + 2 * lane + 1];
      const float mx = warp_max(fmaxf(m[j], fmaxf(x0, x1)));
      const float w0 = exp2f(x0 - mx), w1 = exp2f(x1 - mx), c = exp2f(m[j] - mx);
      l[j] = l[j] * c + warp_sum(w0 + w1);
      m[j] = mx;
      uint32_t hi, lo;
      rc_split(w0, w1, hi, lo);
      *(uint32_t*)(ps + r * LM_PLD + 2 * lane) = hi;
      *(uint32_t*)(ps + (16 + r) * LM_PLD + 2 * lane) = lo;
      if (lane == 0) corr[r] = c;
    }
    __syncthreads();
    const float c0 = corr[ra], c1 = corr[ra + 8];
#pragma unroll
    for (int i = 0; i < 2 * NP; i++) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
#pragma unroll
    for (int k4 = 0; k4 < LM_KEYS / 16; k4++) {
      uint32_t ah[4], al[4];
      rc_ldm(ah, rc_a(ps, LM_PLD, 0, k4 * 16, lane));
      rc_ldm(al, rc_a(ps + 16 * LM_PLD, LM_PLD, 0, k4 * 16, lane));
#pragma unroll
      for (int n = 0; n < NP; n++)
        if (col0 + n * 16 < p.Cp) {
          uint32_t b[4];
          rc_ldmt(b, rc_bk(kb, ld, k4 * 16, col0 + n * 16, lane));
          rc_mma(o[2 * n], ah, b[0], b[1]);
          rc_mma(o[2 * n + 1], ah, b[2], b[3]);
          rc_mma(o[2 * n], al, b[0], b[1]);
          rc_mma(o[2 * n + 1], al, b[2], b[3]);
        }
    }
    __syncthreads();   // the tile and the weights are read
  }
  float* dst = part_of(p, part, splits, row, blockIdx.x) + (size_t)h0 * p.Cp;
#pragma unroll
  for (int i = 0; i < 2 * NP; i++) {
    const int c = col0 + i * 8 + ca;
    if (c < p.Cp) {
      if (ra < nh) *(float2*)(dst + (size_t)ra * p.Cp + c) = make_float2(o[i][0], o[i][1]);
      if (ra + 8 < nh) *(float2*)(dst + (size_t)(ra + 8) * p.Cp + c) = make_float2(o[i][2], o[i][3]);
    }
  }
  if (lane < 2 && warp * 2 + lane < nh)   // maxima in the exponential's own base
    stat_of(p, part, splits, gridDim.z, row, blockIdx.x)[h0 + warp * 2 + lane] =
        make_float2((lane ? m[1] : m[0]) * 0.6931471805599453f, lane ? l[1] : l[0]);
}

// ---- ranges merged, values, gate -----------------------------------------------------------------
// Block (16 value rows, head, row): two rows a warp, whose weights are fetched before the partials are there.
constexpr int LF_PRE = 2;
template <typename KT, typename OT>
__global__ void __launch_bounds__(LA_THREADS) latent_fold_kernel(const __grid_constant__ LatentP p,
                                                                 const float* __restrict__ part, int splits, int rows,
                                                                 const float* __restrict__ proj, long long ld,
                                                                 OT* __restrict__ act, long long lda,
                                                                 const unsigned* d_pos, int pos0) {
  constexpr int CE = Vec16<KT>::N;
  extern __shared__ __align__(16) float sm[];
  float* c = sm;                 // [Cp]
  float* w = c + p.Cp;           // [splits]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, row = blockIdx.z;
  const int e0 = blockIdx.x * LA_EROWS + warp * 2, chunks = p.Cp / CE;
  const KT* W = (const KT*)p.ukv + ((size_t)p.H * p.Dp + (size_t)h * p.Ep) * p.Cp;
  uint4 wv[2][LF_PRE];
#pragma unroll
  for (int j = 0; j < 2; j++)
#pragma unroll
    for (int i = 0; i < LF_PRE; i++) {
      const int k = lane + 32 * i;
      wv[j][i] = e0 + j < p.E && k < chunks ? *(const uint4*)(W + (size_t)(e0 + j) * p.Cp + k * CE) : make_uint4(0, 0, 0, 0);
    }
  const int active = latent_range(p, pos_of(d_pos, pos0, row), splits).active;
  pdl_wait();
  pdl_launch_dependents();
  float gate[2] = {0.f, 0.f};
  if (p.og >= 0 && lane == 0)
#pragma unroll
    for (int j = 0; j < 2; j++)
      if (e0 + j < p.E) gate[j] = proj[(size_t)row * ld + p.og + (size_t)h * p.E + e0 + j];
  const float2* stat = (const float2*)(part + (size_t)rows * splits * p.H * p.Cp) + (size_t)row * splits * p.H + h;
  if (warp == 0) {
    float m = -3.0e38f;
    for (int s = lane; s < active; s += 32) m = fmaxf(m, stat[(size_t)s * p.H].x);
    m = warp_max(m);
    float l = 0.f;
    for (int s = lane; s < active; s += 32) {
      const float2 v = stat[(size_t)s * p.H];
      const float x = expf(v.x - m);
      w[s] = x;
      l = fmaf(x, v.y, l);
    }
    l = 1.0f / warp_sum(l);
    for (int s = lane; s < active; s += 32) w[s] *= l;
  }
  __syncthreads();
  const float* src = part_of(p, part, splits, row, 0) + (size_t)h * p.Cp;
  const size_t step = (size_t)p.H * p.Cp;
  for (int i = tid * 2; i < p.Cp; i += LA_THREADS * 2) {
    float2 a = make_float2(0.f, 0.f);
    for (int s0 = 0; s0 < active; s0 += 16) {
      float2 v[16];
#pragma unroll
      for (int k = 0; k < 16; k++)
        v[k] = s0 + k < active ? *(const float2*)(src + (size_t)(s0 + k) * step + i) : make_float2(0.f, 0.f);
#pragma unroll
      for (int k = 0; k < 16; k++) {
        const float x = s0 + k < active ? w[s0 + k] : 0.f;
        a.x = fmaf(x, v[k].x, a.x);
        a.y = fmaf(x, v[k].y, a.y);
      }
    }
    c[i] = a.x;
    c[i + 1] = a.y;
  }
  __syncthreads();
  float acc[2] = {0.f, 0.f};
  auto dot = [&](const uint4& x, int k, float& s) {
    float f[CE];
    widen16(x, f, (const KT*)nullptr);
#pragma unroll
    for (int e = 0; e < CE; e += 4) {
      const float4 v = *(const float4*)(c + k * CE + e);
      s = fmaf(f[e], v.x, fmaf(f[e + 1], v.y, fmaf(f[e + 2], v.z, fmaf(f[e + 3], v.w, s))));
    }
  };
#pragma unroll
  for (int j = 0; j < 2; j++) {
#pragma unroll
    for (int i = 0; i < LF_PRE; i++)
      if (lane + 32 * i < chunks) dot(wv[j][i], lane + 32 * i, acc[j]);
    for (int k = lane + 32 * LF_PRE; k < chunks; k += 32)
      if (e0 + j < p.E) dot(*(const uint4*)(W + (size_t)(e0 + j) * p.Cp + k * CE), k, acc[j]);
    const float v = warp_sum(acc[j]) * p.out_scale;
    if (lane == 0 && e0 + j < p.E)
      put(act + (size_t)row * lda + p.oa + (size_t)h * p.E + e0 + j, p.og >= 0 ? v * sigmoid_f(gate[j]) : v);
  }
}

// ---- prompt pass on tiles: rotated queries as bf16 -------------------------------------------------
__global__ void __launch_bounds__(LA_THREADS) latent_q_rows_kernel(const __grid_constant__ LatentP p,
                                                                   const float* __restrict__ q, long long ldq,
                                                                   __nv_bfloat16* __restrict__ out, int pos0) {
  __shared__ float2 cs[MX_PAIRS];
  pdl_wait();
  rot_row_table(p, pos0 + blockIdx.x, cs);
  pdl_launch_dependents();
  __syncthreads();
  const float* src = q + (size_t)blockIdx.x * ldq;
  const int w = p.qw(), n = p.H * w;
  __nv_bfloat16* dst = out + (size_t)blockIdx.x * n;
  for (int i = threadIdx.x * 4; i < n; i += LA_THREADS * 4) {   // parts are multiples of 8
    const int d = i % w - p.Dp;
    float4 v = *(const float4*)(src + i);
    if (d >= 0) {
      const float2 a = cs[d >> 1], b = cs[(d >> 1) + 1];
      v = make_float4(d < p.R ? v.x * a.x - v.y * a.y : 0.f, d < p.R ? v.y * a.x + v.x * a.y : 0.f,
                      d + 2 < p.R ? v.z * b.x - v.w * b.y : 0.f, d + 2 < p.R ? v.w * b.x + v.z * b.y : 0.f);
    }
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *(uint2*)(dst + i) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
  }
}

bool mma_fits(const LatentP& p) { return p.Cp <= 512 && LmSmem(p.row()).total <= 220 * 1024; }

template <int NP>
int attend_mma(const LatentP& p, const void* qa, float* part, int rows, int splits, const unsigned* d_pos, int pos0,
               cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(latent_attend_mma_kernel<NP>, 220 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3(splits, (p.H + 15) / 16, rows), dim3(LA_THREADS), LmSmem(p.row()).total, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_attend_mma_kernel<NP>, p, (const __nv_bfloat16*)qa, part, splits, d_pos, pos0));
  return TLB_OK;
}
template <typename KT, int RM>
int attend_any(const LatentP& p, const void* qa, float* part, int rows, int splits, const unsigned* d_pos, int pos0,
               cudaStream_t s) {
  const int values = p.Cp < LA_VALUES ? p.Cp : LA_VALUES;
  const size_t smem = (size_t)(RM * (p.row() + values + MX_TK) + 3 * RM + 32) * sizeof(float);
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(latent_attend_kernel<KT, RM>, 200 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3(splits, (p.H + RM - 1) / RM, rows), dim3(LA_THREADS), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_attend_kernel<KT, RM>, p, (const KT*)qa, part, splits, d_pos, pos0));
  return TLB_OK;
}
template <typename KT, typename OT>
int fold_t(const LatentP& p, const float* part, int splits, const float* proj, long long ld, void* act, long long lda,
           int rows, const unsigned* d_pos, int pos0, cudaStream_t s) {
  LaunchCfg lc(dim3((p.E + LA_EROWS - 1) / LA_EROWS, p.H, rows), dim3(LA_THREADS), (size_t)(p.Cp + splits) * sizeof(float),
               s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_fold_kernel<KT, OT>, p, part, splits, rows, proj, ld, (OT*)act, lda, d_pos, pos0));
  return TLB_OK;
}

}  // namespace

// key ranges of `rows` positions: enough blocks for the SMs, at most the ranges the fold was sized for
int latent_splits(const LatentP& p, int rows) {
  const int n = (p.splits + rows - 1) / rows;
  return n < 1 ? 1 : n;
}
size_t latent_part_floats(const LatentP& p, int rows, int splits) { return (size_t)rows * splits * p.H * (p.Cp + 2); }

int latent_prep_launch(const LatentP& p, const float* proj, long long ld, int rows, int pos0, void* qlat, bool bf16,
                       cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(LA_THREADS), 0, s, pdl_enabled());
  if (bf16)
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_prep_kernel<__nv_bfloat16>, p, proj, ld, pos0, (__nv_bfloat16*)qlat));
  else
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_prep_kernel<float>, p, proj, ld, pos0, (float*)qlat));
  return TLB_OK;
}

int latent_absorb_launch(const LatentP& p, const float* q, long long ldq, const float* proj, void* qa, int rows,
                         const unsigned* d_pos, int pos0, bool bf16, cudaStream_t s) {
  const int slices = (p.Cp + LA_COLS - 1) / LA_COLS + (d_pos && p.owner ? 1 : 0);
  LaunchCfg lc(dim3(slices, p.H, rows), dim3(LA_THREADS), 0, s, pdl_enabled());
  if (bf16)
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_absorb_kernel<__nv_bfloat16>, p, q, ldq, proj, (__nv_bfloat16*)qa, d_pos, pos0));
  else
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_absorb_kernel<float>, p, q, ldq, proj, (float*)qa, d_pos, pos0));
  return TLB_OK;
}

int latent_attend_launch(const LatentP& p, const void* qa, float* part, int rows, int splits, const unsigned* d_pos,
                         int pos0, bool bf16, cudaStream_t s) {
  if (bf16 && mma_fits(p)) {
    if (p.Cp <= 128) return attend_mma<1>(p, qa, part, rows, splits, d_pos, pos0, s);
    if (p.Cp <= 256) return attend_mma<2>(p, qa, part, rows, splits, d_pos, pos0, s);
    return attend_mma<4>(p, qa, part, rows, splits, d_pos, pos0, s);
  }
  if (bf16) return attend_any<__nv_bfloat16, 4>(p, qa, part, rows, splits, d_pos, pos0, s);
  return attend_any<float, 4>(p, qa, part, rows, splits, d_pos, pos0, s);
}

int latent_fold_launch(const LatentP& p, const float* part, int splits, const float* proj, long long ld, void* act,
                       long long lda, int rows, const unsigned* d_pos, int pos0, bool bf16, bool act_bf16,
                       cudaStream_t s) {
  using B = __nv_bfloat16;
  if (bf16)
    return act_bf16 ? fold_t<B, B>(p, part, splits, proj, ld, act, lda, rows, d_pos, pos0, s)
                    : fold_t<B, float>(p, part, splits, proj, ld, act, lda, rows, d_pos, pos0, s);
  return fold_t<float, float>(p, part, splits, proj, ld, act, lda, rows, d_pos, pos0, s);
}

int latent_q_rows_launch(const LatentP& p, const float* q, long long ldq, void* out, int rows, int pos0, cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(LA_THREADS), 0, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, latent_q_rows_kernel, p, q, ldq, (__nv_bfloat16*)out, pos0));
  return TLB_OK;
}

}  // namespace tlb
