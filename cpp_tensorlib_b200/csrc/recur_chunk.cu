// The recurrences of a prompt pass in chunks of 64 tokens on the tensor pipe (bf16 models; widths that
// are multiples of 8, state width up to 128).  With b_t the running sum of log decays inside a chunk and
// S the state in front of it, both recurrences are
//   O_t = exp(b_t) q_t S + sum_{s <= t} exp(b_t - b_s) (q_t . k_s) u_s
//   S  <- exp(b_L) S + sum_s exp(b_L - b_s) k_s u_s^T
// with u_s = dt_s x_s for ssd, and for the delta rule U = T (V - exp(b) (K S)), where
// T = (I + A)^-1 diag(beta), A_ts = beta_t exp(b_t - b_s) (k_t . k_s) below the diagonal
// (the chunk-parallel form of DeltaNet, Yang et al., "Parallelizing Linear Transformers with the Delta
// Rule over Sequence Length").
//
// What the short convolutions leave (q, k, v) is bf16 and enters the products exactly; everything else
// -- unit norms, step sizes, decays, T, U, the state -- is f32: as factors of rows and columns outside
// the products, or as operands split into two bf16 planes (hi + lo).  The state stays in f32
// accumulators for the whole pass.
//
//   delta_solve   (chunk, head): T of every chunk, in two planes
//   recur_chunk   (32 value columns, head): the chunks in order
#include "mixers.cuh"
#include "rows_mma.cuh"

namespace tlb {

namespace {

constexpr int RC_L = 64, RC_E = 32, RC_THREADS = 128;
constexpr int RC_TLD = RC_L + 8, RC_ELD = RC_E + 8;

// b_t of the chunk (lanes hold tokens lane and lane + 32) from the rates x_t = -log g_t
__device__ __forceinline__ void rc_scan(float x0, float x1, float& b0, float& b1) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float y0 = __shfl_up_sync(0xffffffffu, x0, o), y1 = __shfl_up_sync(0xffffffffu, x1, o);
    if (lane >= o) { x0 += y0; x1 += y1; }
  }
  x1 += __shfl_sync(0xffffffffu, x0, 31);
  b0 = -x0;
  b1 = -x1;
}

// ---- T of one chunk and head -----------------------------------------------------------------
template <int DP>
__global__ void __launch_bounds__(RC_THREADS) delta_solve_kernel(const __grid_constant__ RecurP p,
                                                                 const __nv_bfloat16* __restrict__ conv,
                                                                 const float2* __restrict__ gates,
                                                                 const float2* __restrict__ norms,
                                                                 __nv_bfloat16* __restrict__ T, int rows) {
  constexpr int LD = DP + 8, AL = RC_L + 1;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* ks = (__nv_bfloat16*)smem;              // [64][LD]
  float* A = (float*)(smem + (size_t)RC_L * LD * 2);     // [64][AL]
  float* X = A + RC_L * AL;                              // [64][AL]
  float* P = X + RC_L * AL;                              // [3][16][17]
  __shared__ float sb[RC_L], sbeta[RC_L], sn[RC_L];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = blockIdx.x * RC_L, h = blockIdx.y, kg = h / (p.H / p.G), n = rows - t0 < RC_L ? rows - t0 : RC_L;
  for (int i = tid; i < RC_L * LD / 8; i += RC_THREADS) ((uint4*)ks)[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < RC_L * AL; i += RC_THREADS) X[i] = 0.f;
  pdl_wait();
  pdl_launch_dependents();
  __syncthreads();
  const int dch = p.D / 8;
  for (int i = tid; i < n * dch; i += RC_THREADS) {
    const int r = i / dch, c = i - r * dch;
    *(uint4*)(ks + r * LD + c * 8) = *(const uint4*)(conv + (size_t)(t0 + r) * p.cv.C + p.ck + kg * p.D + c * 8);
  }
  if (warp == 0) {
    const float2 z = make_float2(0.f, 0.f);
    const float2 g0 = lane < n ? gates[(size_t)(t0 + lane) * p.H + h] : z;
    const float2 g1 = lane + 32 < n ? gates[(size_t)(t0 + lane + 32) * p.H + h] : z;
    float b0, b1;
    rc_scan(g0.y, g1.y, b0, b1);
    sb[lane] = b0; sb[lane + 32] = b1;
    sbeta[lane] = g0.x; sbeta[lane + 32] = g1.x;
    sn[lane] = lane < n ? norms[(size_t)(t0 + lane) * p.G + kg].y : 0.f;
    sn[lane + 32] = lane + 32 < n ? norms[(size_t)(t0 + lane + 32) * p.G + kg].y : 0.f;
  }
  __syncthreads();
  float s[8][4];
#pragma unroll
  for (int i = 0; i < 8; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
  for (int k = 0; k < DP; k += 16) {
    uint32_t a[4], b[4];
    rc_ldm(a, rc_a(ks, LD, warp * 16, k, lane));
#pragma unroll
    for (int j = 0; j < 4; j++) {
      rc_ldm(b, rc_bn(ks, LD, j * 16, k, lane));
      rc_mma(s[2 * j], a, b[0], b[1]);
      rc_mma(s[2 * j + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int j = 0; j < 8; j++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int t = warp * 16 + (lane >> 2) + (e >> 1) * 8, c = j * 8 + (lane & 3) * 2 + (e & 1);
      A[t * AL + c] = c < t ? s[j][e] * sn[t] * sn[c] * sbeta[t] * expf(sb[t] - sb[c]) : 0.f;
    }
  __syncthreads();
  // (I + A)^-1 in blocks of 16: the diagonal blocks column by column, then the blocks below, one
  // block diagonal after the other: X_ij = -X_ii sum_{j <= k < i} A_ik X_kj
  if (tid < 64) {
    const int o = (tid >> 4) * 16, c = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; i++) {
      float v = i == c ? 1.f : 0.f;
#pragma unroll
      for (int k = 0; k < i; k++) v = fmaf(-A[(o + i) * AL + o + k], x[k], v);
      x[i] = v;
    }
#pragma unroll
    for (int i = 0; i < 16; i++) X[(o + i) * AL + o + c] = x[i];
  }
  for (int d = 1; d < 4; d++) {
    __syncthreads();
    for (int i = tid; i < (4 - d) * 256; i += RC_THREADS) {
      const int blk = i >> 8, r = (i >> 4) & 15, c = i & 15, bi = blk + d, bj = blk;
      float v = 0.f;
      for (int k = bj * 16; k < bi * 16; k++) v = fmaf(A[(bi * 16 + r) * AL + k], X[k * AL + bj * 16 + c], v);
      P[(blk * 16 + r) * 17 + c] = v;
    }
    __syncthreads();
    for (int i = tid; i < (4 - d) * 256; i += RC_THREADS) {
      const int blk = i >> 8, r = (i >> 4) & 15, c = i & 15, bi = blk + d, bj = blk;
      float v = 0.f;
#pragma unroll
      for (int k = 0; k < 16; k++) v = fmaf(X[(bi * 16 + r) * AL + bi * 16 + k], P[(blk * 16 + k) * 17 + c], v);
      X[(bi * 16 + r) * AL + bj * 16 + c] = -v;
    }
  }
  __syncthreads();
  __nv_bfloat16* out = T + ((size_t)blockIdx.x * p.H + h) * 2 * RC_L * RC_L;
  for (int i = tid; i < RC_L * RC_L / 2; i += RC_THREADS) {
    const int r = i / (RC_L / 2), c = (i % (RC_L / 2)) * 2;
    uint32_t hi, lo;
    rc_split(X[r * AL + c] * sbeta[c], X[r * AL + c + 1] * sbeta[c + 1], hi, lo);
    ((uint32_t*)out)[i] = hi;
    ((uint32_t*)(out + RC_L * RC_L))[i] = lo;
  }
}

// ---- the chunks of one head and 32 value columns -----------------------------------------------
template <int DP, bool DELTA>
struct RcSmem {
  static constexpr int LD = DP + 8;
  static constexpr size_t K = 0;                                            // [2][64][LD]
  static constexpr size_t Q = K + (size_t)2 * RC_L * LD * 2;
  static constexpr size_t X = Q + (size_t)2 * RC_L * LD * 2;                // [2][64][ELD]
  static constexpr size_t S = X + (size_t)2 * RC_L * RC_ELD * 2;            // [2 planes][DP][ELD]
  static constexpr size_t W = S + (size_t)2 * DP * RC_ELD * 2;              // [2 planes][64][ELD]
  static constexpr size_t U = W + (size_t)2 * RC_L * RC_ELD * 2;            // delta: [2 planes][64][ELD]
  static constexpr size_t T = U + (DELTA ? (size_t)2 * RC_L * RC_ELD * 2 : 0);   // delta: [2][2 planes][64][TLD]
  static constexpr size_t SC = T + (DELTA ? (size_t)4 * RC_L * RC_TLD * 2 : 0);  // [4][64] f32
  static constexpr size_t TOTAL = SC + 4 * RC_L * 4;
};

template <int DP, bool DELTA>
__global__ void __launch_bounds__(RC_THREADS, DELTA ? 1 : 2)
    recur_chunk_kernel(const __grid_constant__ RecurP p, const __nv_bfloat16* __restrict__ conv,
                       const float2* __restrict__ gates, const float2* __restrict__ norms,
                       const __nv_bfloat16* __restrict__ T, float* __restrict__ o, int rows, int pos0) {
  using SM = RcSmem<DP, DELTA>;
  constexpr int LD = SM::LD, MT = DP / 64;      // state row tiles of 16 per warp
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* ksm = (__nv_bfloat16*)(smem + SM::K);
  __nv_bfloat16* qsm = (__nv_bfloat16*)(smem + SM::Q);
  __nv_bfloat16* xsm = (__nv_bfloat16*)(smem + SM::X);
  __nv_bfloat16* ssm = (__nv_bfloat16*)(smem + SM::S);
  __nv_bfloat16* wsm = (__nv_bfloat16*)(smem + SM::W);
  __nv_bfloat16* usm = (__nv_bfloat16*)(smem + SM::U);
  __nv_bfloat16* tsm = (__nv_bfloat16*)(smem + SM::T);
  float* sb = (float*)(smem + SM::SC);          // b_t
  float* sg = sb + RC_L;                        // dt_s of ssd
  float* snk = sg + RC_L;                       // 1 / |k_s|
  float* snq = snk + RC_L;                      // D^-1/2 / |q_t|
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wr = warp * 16;
  const int h = blockIdx.y, c0 = blockIdx.x * RC_E, kg = h / (p.H / p.G), D = p.D, E = p.E;
  const int nch = (rows + RC_L - 1) / RC_L, dch = D / 8, ech = (E - c0 < RC_E ? E - c0 : RC_E) / 8;
  for (int i = tid; i < (int)(SM::SC / 16); i += RC_THREADS) ((uint4*)smem)[i] = make_uint4(0, 0, 0, 0);
  pdl_wait();
  pdl_launch_dependents();
  __syncthreads();
  auto fetch = [&](int ch, int buf) {
    const int t0 = ch * RC_L, n = rows - t0 < RC_L ? rows - t0 : RC_L;
    for (int i = tid; i < RC_L * dch; i += RC_THREADS) {
      const int r = i / dch, c = i - r * dch;
      const bool on = r < n;
      const __nv_bfloat16* row = conv + (size_t)(on ? t0 + r : t0) * p.cv.C + kg * D + c * 8;
      rc_cp16(ksm + (buf * RC_L + r) * LD + c * 8, row + p.ck, on);
      rc_cp16(qsm + (buf * RC_L + r) * LD + c * 8, row + p.cq, on);
    }
    for (int i = tid; i < RC_L * ech; i += RC_THREADS) {
      const int r = i / ech, c = i - r * ech;
      const bool on = r < n;
      rc_cp16(xsm + (buf * RC_L + r) * RC_ELD + c * 8, conv + (size_t)(on ? t0 + r : t0) * p.cv.C + p.cvv + h * E + c0 + c * 8, on);
    }
    if (DELTA) {
      const __nv_bfloat16* src = T + ((size_t)ch * p.H + h) * 2 * RC_L * RC_L;
      for (int i = tid; i < 2 * RC_L * 8; i += RC_THREADS)
        rc_cp16(tsm + ((size_t)buf * 2 * RC_L + (i >> 3)) * RC_TLD + (i & 7) * 8, src + (size_t)i * 8, true);
    }
  };
  // warp 0 carries the next chunk's scalars in registers (tokens lane and lane + 32)
  float2 g0, g1, n0, n1;
  auto scalars = [&](int ch) {
    const int t0 = ch * RC_L + lane, t1 = t0 + 32;
    const float2 z = make_float2(0.f, 0.f);
    g0 = t0 < rows ? gates[(size_t)t0 * p.H + h] : z;
    g1 = t1 < rows ? gates[(size_t)t1 * p.H + h] : z;
    if (DELTA) {
      n0 = t0 < rows ? norms[(size_t)t0 * p.G + kg] : z;
      n1 = t1 < rows ? norms[(size_t)t1 * p.G + kg] : z;
    }
  };
  // state: this warp's rows of it, 32 columns, as accumulators
  float s[MT][4][4];
  float* S = p.S + (size_t)h * D * E;
  auto state_at = [&](int mt, int nt, int e, int& r, int& c) {
    r = (warp * MT + mt) * 16 + (lane >> 2) + (e >> 1) * 8;
    c = c0 + nt * 8 + (lane & 3) * 2 + (e & 1);
  };
#pragma unroll
  for (int mt = 0; mt < MT; mt++)
#pragma unroll
    for (int nt = 0; nt < 4; nt++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        int r, c;
        state_at(mt, nt, e, r, c);
        s[mt][nt][e] = pos0 > 0 && r < D && c < E ? S[(size_t)r * E + c] : 0.f;
      }
  fetch(0, 0);
  rc_commit();
  if (warp == 0) scalars(0);
  for (int ch = 0; ch < nch; ch++) {
    const int buf = ch & 1, t0 = ch * RC_L, n = rows - t0 < RC_L ? rows - t0 : RC_L;
    // the state in front of the chunk, in two planes, for the products below
#pragma unroll
    for (int mt = 0; mt < MT; mt++)
#pragma unroll
      for (int nt = 0; nt < 4; nt++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          uint32_t hi, lo;
          rc_split(s[mt][nt][2 * e], s[mt][nt][2 * e + 1], hi, lo);
          const int at = ((warp * MT + mt) * 16 + (lane >> 2) + e * 8) * RC_ELD + nt * 8 + (lane & 3) * 2;
          *(uint32_t*)(ssm + at) = hi;
          *(uint32_t*)(ssm + DP * RC_ELD + at) = lo;
        }
    if (warp == 0) {
      float b0, b1;
      rc_scan(g0.y, g1.y, b0, b1);
      sb[lane] = b0; sb[lane + 32] = b1;
      sg[lane] = g0.x; sg[lane + 32] = g1.x;
      if (DELTA) { snk[lane] = n0.y; snk[lane + 32] = n1.y; snq[lane] = n0.x; snq[lane + 32] = n1.x; }
      if (ch + 1 < nch) scalars(ch + 1);
    }
    rc_wait<0>();
    __syncthreads();
    if (ch + 1 < nch) {
      fetch(ch + 1, buf ^ 1);
      rc_commit();
    }
    const __nv_bfloat16 *K = ksm + buf * RC_L * LD, *Q = qsm + buf * RC_L * LD, *X = xsm + buf * RC_L * RC_ELD;
    const int ra = wr + (lane >> 2), cb = (lane & 3) * 2;     // the thread's rows are ra and ra + 8
    const float ba = sb[ra], bb = sb[ra + 8], bL = sb[RC_L - 1];
    // q S, k S (both planes of S), q k^T for the rows of this warp
    float qs[4][4], kS[4][4], m[8][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int e = 0; e < 4; e++) qs[i][e] = kS[i][e] = m[i][e] = m[i + 4][e] = 0.f;
#pragma unroll
    for (int k = 0; k < DP; k += 16) {
      uint32_t aq[4], ak[4];
      rc_ldm(aq, rc_a(Q, LD, wr, k, lane));
      if (DELTA) rc_ldm(ak, rc_a(K, LD, wr, k, lane));
#pragma unroll
      for (int pl = 0; pl < 2; pl++)
#pragma unroll
        for (int j = 0; j < 2; j++) {
          uint32_t b[4];
          rc_ldmt(b, rc_bk(ssm + pl * DP * RC_ELD, RC_ELD, k, j * 16, lane));
          rc_mma(qs[2 * j], aq, b[0], b[1]);
          rc_mma(qs[2 * j + 1], aq, b[2], b[3]);
          if (DELTA) {
            rc_mma(kS[2 * j], ak, b[0], b[1]);
            rc_mma(kS[2 * j + 1], ak, b[2], b[3]);
          }
        }
#pragma unroll
      for (int j = 0; j < 4; j++)
        if (j <= warp) {
          uint32_t b[4];
          rc_ldm(b, rc_bn(K, LD, j * 16, k, lane));
          rc_mma(m[2 * j], aq, b[0], b[1]);
          rc_mma(m[2 * j + 1], aq, b[2], b[3]);
        }
    }
    // decays (and unit norms, step sizes) of q k^T, then as operand planes
    uint32_t mh[4][4], ml[4][4];
    const float qa = DELTA ? snq[ra] : 1.f, qb = DELTA ? snq[ra + 8] : 1.f;
#pragma unroll
    for (int j = 0; j < 8; j++) {
      float w[4];
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int c = j * 8 + cb + (e & 1), t = e < 2 ? ra : ra + 8;
        const float f = c <= t ? expf((e < 2 ? ba : bb) - sb[c]) * (DELTA ? snk[c] * (e < 2 ? qa : qb) : sg[c]) : 0.f;
        w[e] = j <= 2 * warp + 1 ? m[j][e] * f : 0.f;
      }
      rc_split(w[0], w[1], mh[j >> 1][(j & 1) * 2], ml[j >> 1][(j & 1) * 2]);
      rc_split(w[2], w[3], mh[j >> 1][(j & 1) * 2 + 1], ml[j >> 1][(j & 1) * 2 + 1]);
    }
    if (DELTA) {
      // R = v - exp(b) |k|^-1 (k S), in planes
      const float fa = expf(ba) * snk[ra], fb = expf(bb) * snk[ra + 8];
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int at = (ra + 8 * e) * RC_ELD + j * 8 + cb;
          const uint32_t v = *(const uint32_t*)(X + at);
          const float f = e ? fb : fa;
          uint32_t hi, lo;
          rc_split(fmaf(-f, kS[j][2 * e], __uint_as_float(v << 16)),
                   fmaf(-f, kS[j][2 * e + 1], __uint_as_float(v & 0xffff0000u)), hi, lo);
          *(uint32_t*)(usm + at) = hi;
          *(uint32_t*)(usm + RC_L * RC_ELD + at) = lo;
        }
      __syncthreads();
      float u[4][4];
#pragma unroll
      for (int i = 0; i < 4; i++) u[i][0] = u[i][1] = u[i][2] = u[i][3] = 0.f;
      const __nv_bfloat16* Tp = tsm + (size_t)buf * 2 * RC_L * RC_TLD;
#pragma unroll
      for (int k = 0; k < 4; k++)
        if (k <= warp) {
          uint32_t ah[4], al[4];
          rc_ldm(ah, rc_a(Tp, RC_TLD, wr, k * 16, lane));
          rc_ldm(al, rc_a(Tp + RC_L * RC_TLD, RC_TLD, wr, k * 16, lane));
#pragma unroll
          for (int j = 0; j < 2; j++) {
            uint32_t bh[4], bl[4];
            rc_ldmt(bh, rc_bk(usm, RC_ELD, k * 16, j * 16, lane));
            rc_ldmt(bl, rc_bk(usm + RC_L * RC_ELD, RC_ELD, k * 16, j * 16, lane));
            rc_mma(u[2 * j], ah, bh[0], bh[1]); rc_mma(u[2 * j + 1], ah, bh[2], bh[3]);
            rc_mma(u[2 * j], ah, bl[0], bl[1]); rc_mma(u[2 * j + 1], ah, bl[2], bl[3]);
            rc_mma(u[2 * j], al, bh[0], bh[1]); rc_mma(u[2 * j + 1], al, bh[2], bh[3]);
          }
        }
      __syncthreads();   // R is read: its planes become U's
      const float ga = expf(bL - ba) * snk[ra], gb = expf(bL - bb) * snk[ra + 8];
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int at = (ra + 8 * e) * RC_ELD + j * 8 + cb;
          const float f = e ? gb : ga;
          uint32_t hi, lo;
          rc_split(u[j][2 * e], u[j][2 * e + 1], hi, lo);
          *(uint32_t*)(usm + at) = hi;
          *(uint32_t*)(usm + RC_L * RC_ELD + at) = lo;
          rc_split(u[j][2 * e] * f, u[j][2 * e + 1] * f, hi, lo);
          *(uint32_t*)(wsm + at) = hi;
          *(uint32_t*)(wsm + RC_L * RC_ELD + at) = lo;
        }
    } else {
      const float ga = expf(bL - ba) * sg[ra], gb = expf(bL - bb) * sg[ra + 8];
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int at = (ra + 8 * e) * RC_ELD + j * 8 + cb;
          const uint32_t v = *(const uint32_t*)(X + at);
          const float f = e ? gb : ga;
          uint32_t hi, lo;
          rc_split(f * __uint_as_float(v << 16), f * __uint_as_float(v & 0xffff0000u), hi, lo);
          *(uint32_t*)(wsm + at) = hi;
          *(uint32_t*)(wsm + RC_L * RC_ELD + at) = lo;
        }
    }
    __syncthreads();
    // O = exp(b) (q S) + M U
    const float ea = expf(ba) * qa, eb = expf(bb) * qb;
#pragma unroll
    for (int j = 0; j < 4; j++) { qs[j][0] *= ea; qs[j][1] *= ea; qs[j][2] *= eb; qs[j][3] *= eb; }
    const __nv_bfloat16* Up = DELTA ? usm : X;
#pragma unroll
    for (int k = 0; k < 4; k++)
      if (k <= warp) {
#pragma unroll
        for (int j = 0; j < 2; j++) {
          uint32_t b[4];
          rc_ldmt(b, rc_bk(Up, RC_ELD, k * 16, j * 16, lane));
          rc_mma(qs[2 * j], mh[k], b[0], b[1]); rc_mma(qs[2 * j + 1], mh[k], b[2], b[3]);
          rc_mma(qs[2 * j], ml[k], b[0], b[1]); rc_mma(qs[2 * j + 1], ml[k], b[2], b[3]);
          if (DELTA) {
            rc_ldmt(b, rc_bk(usm + RC_L * RC_ELD, RC_ELD, k * 16, j * 16, lane));
            rc_mma(qs[2 * j], mh[k], b[0], b[1]); rc_mma(qs[2 * j + 1], mh[k], b[2], b[3]);
          }
        }
      }
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int t = ra + 8 * e;
      if (t < n) {
        float* dst = o + ((size_t)(t0 + t) * p.H + h) * E + c0;
#pragma unroll
        for (int j = 0; j < 4; j++)
          if (j < ech) *(float2*)(dst + j * 8 + cb) = make_float2(qs[j][2 * e], qs[j][2 * e + 1]);
      }
    }
    // S = exp(b_L) S + K^T (weighted U)
    const float eL = expf(bL);
#pragma unroll
    for (int mt = 0; mt < MT; mt++)
#pragma unroll
      for (int nt = 0; nt < 4; nt++)
#pragma unroll
        for (int e = 0; e < 4; e++) s[mt][nt][e] *= eL;
#pragma unroll
    for (int k = 0; k < 4; k++) {
      uint32_t a[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; mt++) rc_ldmt(a[mt], rc_at(K, LD, (warp * MT + mt) * 16, k * 16, lane));
#pragma unroll
      for (int pl = 0; pl < 2; pl++)
#pragma unroll
        for (int j = 0; j < 2; j++) {
          uint32_t b[4];
          rc_ldmt(b, rc_bk(wsm + pl * RC_L * RC_ELD, RC_ELD, k * 16, j * 16, lane));
#pragma unroll
          for (int mt = 0; mt < MT; mt++) {
            rc_mma(s[mt][2 * j], a[mt], b[0], b[1]);
            rc_mma(s[mt][2 * j + 1], a[mt], b[2], b[3]);
          }
        }
    }
    __syncthreads();   // the chunk's operands and planes are read: the next one may overwrite them
  }
#pragma unroll
  for (int mt = 0; mt < MT; mt++)
#pragma unroll
    for (int nt = 0; nt < 4; nt++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        int r, c;
        state_at(mt, nt, e, r, c);
        if (r < D && c < E) S[(size_t)r * E + c] = s[mt][nt][e];
      }
}

template <int DP, bool DELTA>
int rc_launch(const RecurP& p, const void* conv, const float2* gates, const float2* norms, void* T, float* o, int rows,
              int pos0, cudaStream_t s) {
  if (DELTA) {
    constexpr int smem = RC_L * (DP + 8) * 2 + (2 * RC_L * (RC_L + 1) + 3 * 16 * 17) * 4;
    static std::atomic<unsigned long long> done{0};
    const int rc = ensure_dynamic_smem(delta_solve_kernel<DP>, smem, done);
    if (rc) return rc;
    LaunchCfg lc(dim3((rows + RC_L - 1) / RC_L, p.H), dim3(RC_THREADS), smem, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, delta_solve_kernel<DP>, p, (const __nv_bfloat16*)conv, gates, norms,
                                (__nv_bfloat16*)T, rows));
  }
  constexpr int smem = (int)RcSmem<DP, DELTA>::TOTAL;
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(recur_chunk_kernel<DP, DELTA>, smem, done);
  if (rc) return rc;
  LaunchCfg lc(dim3((p.E + RC_E - 1) / RC_E, p.H), dim3(RC_THREADS), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, recur_chunk_kernel<DP, DELTA>, p, (const __nv_bfloat16*)conv, gates, norms,
                              (const __nv_bfloat16*)T, o, rows, pos0));
  return TLB_OK;
}

}  // namespace

bool recur_chunk_eligible(const RecurP& p) { return p.D <= 128 && p.D % 8 == 0 && p.E % 8 == 0 && p.cv.taps <= 8; }

size_t recur_chunk_scratch_bytes(const RecurP& p, int rows) {
  return p.kind == MIX_DELTA ? (size_t)((rows + RC_L - 1) / RC_L) * p.H * 2 * RC_L * RC_L * 2 : 0;
}

int recur_chunk_launch(const RecurP& p, const void* conv, const float2* gates, const float2* norms, void* scratch,
                       float* o, int rows, int pos0, cudaStream_t s) {
  if (p.kind == MIX_DELTA)
    return p.D <= 64 ? rc_launch<64, true>(p, conv, gates, norms, scratch, o, rows, pos0, s)
                     : rc_launch<128, true>(p, conv, gates, norms, scratch, o, rows, pos0, s);
  return p.D <= 64 ? rc_launch<64, false>(p, conv, gates, norms, scratch, o, rows, pos0, s)
                   : rc_launch<128, false>(p, conv, gates, norms, scratch, o, rows, pos0, s);
}

}  // namespace tlb
