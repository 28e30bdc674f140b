// Gated linear attention of a prompt pass.  Per head, with a decay per key channel,
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t.
// The rates -log a_t of every row come first (gla_rates), f32 throughout.  f32 models then run the
// recurrence token by token (recur_scan_kernel of mixers.cu).  bf16 models run it in chunks of 64 tokens on
// the tensor pipe, with b_t the running sum of rates inside a chunk:
//   gla_state  (chunk, head, value columns)      U = sum_s exp(b_s - b_L) k_s v_s^T, and exp(-b_L)
//   gla_carry  (state elements)                  S <- diag(exp(-b_L)) S + U down the chunks, each chunk's U
//                                                replaced by the state in front of it
//   gla_out    (chunk, head)                     o_t = (exp(-b_t) q_t) S + sum_{s <= t} A_ts v_s,
//                                                A_ts = (exp(-b_t) q_t) . (exp(b_s) k_s)
// All chunks run at once in the first and the last.  Scaled queries and keys, A and S enter the products as
// two bf16 planes (hi + lo); values are bf16.  The factors of A grow as exp(b_L): a chunk with a channel
// that decays below exp(-60) takes every exp(b_s - b_t) by itself instead.
#include "mixers.cuh"
#include "rows_mma.cuh"

namespace tlb {

namespace {

constexpr int GC_L = 64, GC_E = 64, GC_THREADS = 256, GC_ELD = GC_E + 8;   // GC_E: value columns of gla_out
constexpr float GC_MOST = 60.f;   // largest b_L of the factored form

// ---- rates ---------------------------------------------------------------------------------------
constexpr int GR_ROWS = 32, GR_K = 8;
__global__ void __launch_bounds__(256) gla_rates_kernel(const __grid_constant__ RecurP p, const float* __restrict__ proj,
                                                        long long ld, float* __restrict__ rates, int rows) {
  __shared__ float a[GR_ROWS][GR_K];
  const int HD = p.H * p.D, c = blockIdx.x * 256 + threadIdx.x, t0 = blockIdx.y * GR_ROWS;
  const float bias = c < HD ? p.a_bias[c] : 0.f;
  float acc[GR_ROWS];
#pragma unroll
  for (int t = 0; t < GR_ROWS; t++) acc[t] = bias;
  pdl_wait();
  pdl_launch_dependents();
  for (int r0 = 0; r0 < p.rank; r0 += GR_K) {
    __syncthreads();
    {
      const int t = threadIdx.x / GR_K, r = threadIdx.x % GR_K;
      a[t][r] = t0 + t < rows && r0 + r < p.rank ? proj[(size_t)(t0 + t) * ld + p.ob + r0 + r] : 0.f;
    }
    float w[GR_K];
#pragma unroll
    for (int r = 0; r < GR_K; r++) w[r] = c < HD && r0 + r < p.rank ? p.a_up[(size_t)(r0 + r) * HD + c] : 0.f;
    __syncthreads();
#pragma unroll
    for (int t = 0; t < GR_ROWS; t++)
#pragma unroll
      for (int r = 0; r < GR_K; r++) acc[t] = fmaf(a[t][r], w[r], acc[t]);
  }
  if (c >= HD) return;
#pragma unroll
  for (int t = 0; t < GR_ROWS; t++)
    if (t0 + t < rows) rates[(size_t)(t0 + t) * HD + c] = gla_rate(acc[t], p.tau);
}

// the rates of one channel for TG of a chunk's tokens, their sum and the sum of all groups
template <int TG>
__device__ __forceinline__ float load_rates(const float* rates, size_t stride, int n, bool on, float (&x)[TG]) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < TG; i++) {
    x[i] = on && i < n ? rates[(size_t)i * stride] : 0.f;
    s += x[i];
  }
  return s;
}
__device__ __forceinline__ void put_planes(__nv_bfloat16* at, size_t plane, float v) {
  const __nv_bfloat16 hi = __float2bfloat16_rn(v);
  at[0] = hi;
  at[plane] = __float2bfloat16_rn(v - __bfloat162float(hi));
}
// four adjacent elements of a row of which `left` are there; vec: rows start on 16 bytes
__device__ __forceinline__ float4 load4(const float* at, int left, bool vec) {
  if (vec && left >= 4) return *(const float4*)at;
  return make_float4(left > 0 ? at[0] : 0.f, left > 1 ? at[1] : 0.f, left > 2 ? at[2] : 0.f, left > 3 ? at[3] : 0.f);
}
// 64 rows x W columns of f32 rows as bf16; columns from `cols` on and rows from n on are zero
template <int W>
__device__ __forceinline__ void load_values(__nv_bfloat16* vs, const float* src, long long ld, int n, int cols, bool vec) {
#pragma unroll 4
  for (int i = threadIdx.x; i < GC_L * W / 4; i += GC_THREADS) {
    const int t = i / (W / 4), c = (i - t * (W / 4)) * 4;
    const float4 v = load4(src + (size_t)t * ld + c, t < n ? cols - c : 0, vec);
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *(uint2*)(vs + t * (W + 8) + c) = make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
  }
}

// ---- what a chunk adds to the state -----------------------------------------------------------------
template <int DP> constexpr int GS_E = DP <= 128 ? 128 : 64;   // value columns of a block
template <int DP>
__global__ void __launch_bounds__(GC_THREADS) gla_state_kernel(const __grid_constant__ RecurP p,
                                                               const float* __restrict__ proj, long long ld,
                                                               const float* __restrict__ rates, float* __restrict__ U,
                                                               float* __restrict__ decay, int rows) {
  constexpr int LD = DP + 8, NG = GC_THREADS / DP, TG = GC_L / NG, MT = DP >= 128 ? DP / 128 : 1;
  constexpr int SE = GS_E<DP>, SLD = SE + 8, NT = (DP >= 128 ? SE : SE / 2) / 16;   // pairs of column tiles of a warp
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* ks = (__nv_bfloat16*)smem;    // [2 planes][64][LD]
  __nv_bfloat16* vs = ks + 2 * GC_L * LD;      // [64][SLD]
  float* gsum = (float*)(vs + GC_L * SLD);     // [NG][DP]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = p.D, E = p.E;
  const int e0 = blockIdx.x * SE, h = blockIdx.y, ch = blockIdx.z, t0 = ch * GC_L;
  const int n = rows - t0 < GC_L ? rows - t0 : GC_L, d = tid % DP, grp = tid / DP, tg = grp * TG, HD = p.H * D;
  pdl_wait();
  pdl_launch_dependents();
  float x[TG], kv[TG];
  const float* kr = proj + (size_t)(t0 + tg) * ld + p.ck + h * D + d;
#pragma unroll
  for (int i = 0; i < TG; i++) kv[i] = d < D && tg + i < n ? kr[(size_t)i * ld] : 0.f;
  gsum[grp * DP + d] = load_rates<TG>(rates + (size_t)(t0 + tg) * HD + h * D + d, HD, n - tg, d < D, x);
  load_values<SE>(vs, proj + (size_t)t0 * ld + p.cvv + h * E + e0, ld, n, E - e0, (E & 3) == 0);
  __syncthreads();
  float r = 0.f;
  for (int g = grp + 1; g < NG; g++) r += gsum[g * DP + d];
#pragma unroll
  for (int i = TG - 1; i >= 0; i--) {
    put_planes(ks + (tg + i) * LD + d, (size_t)GC_L * LD, kv[i] * expf(-r));
    r += x[i];
  }
  if (blockIdx.x == 0 && grp == 0 && d < D) decay[((size_t)ch * p.H + h) * D + d] = expf(-r);
  __syncthreads();
  const int m0 = DP >= 128 ? warp * MT : warp & 3, n0 = DP >= 128 ? 0 : (warp >> 2) * (SE / 2);
  float u[MT][2 * NT][4];
#pragma unroll
  for (int i = 0; i < MT; i++)
#pragma unroll
    for (int j = 0; j < 2 * NT; j++) u[i][j][0] = u[i][j][1] = u[i][j][2] = u[i][j][3] = 0.f;
#pragma unroll
  for (int k = 0; k < GC_L; k += 16) {
    uint32_t a[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
      for (int pl = 0; pl < 2; pl++) rc_ldmt(a[i][pl], rc_at(ks + pl * GC_L * LD, LD, (m0 + i) * 16, k, lane));
#pragma unroll
    for (int j = 0; j < NT; j++) {
      uint32_t b[4];
      rc_ldmt(b, rc_bk(vs, SLD, k, n0 + j * 16, lane));
#pragma unroll
      for (int i = 0; i < MT; i++)
#pragma unroll
        for (int pl = 0; pl < 2; pl++) {
          rc_mma(u[i][2 * j], a[i][pl], b[0], b[1]);
          rc_mma(u[i][2 * j + 1], a[i][pl], b[2], b[3]);
        }
    }
  }
  float* dst = U + ((size_t)ch * p.H + h) * D * E;
#pragma unroll
  for (int i = 0; i < MT; i++)
#pragma unroll
    for (int j = 0; j < 2 * NT; j++)
#pragma unroll
      for (int f = 0; f < 2; f++) {
        const int dd = (m0 + i) * 16 + (lane >> 2) + f * 8, e = e0 + n0 + j * 8 + (lane & 3) * 2;
        if (dd >= D) continue;
        float* at = dst + (size_t)dd * E + e;
        if ((E & 1) == 0) {
          if (e < E) *(float2*)at = make_float2(u[i][j][2 * f], u[i][j][2 * f + 1]);
        } else {
          if (e < E) at[0] = u[i][j][2 * f];
          if (e + 1 < E) at[1] = u[i][j][2 * f + 1];
        }
      }
}

// ---- the state down the chunks ------------------------------------------------------------------------
constexpr int GA_BATCH = 8;
__device__ __forceinline__ float fma_state(float s, float g, float u) { return fmaf(s, g, u); }
__device__ __forceinline__ float4 fma_state(float4 s, float g, float4 u) {
  return make_float4(fmaf(s.x, g, u.x), fmaf(s.y, g, u.y), fmaf(s.z, g, u.z), fmaf(s.w, g, u.w));
}
template <typename V>   // float4 where four elements share a row of the state
__global__ void __launch_bounds__(256) gla_carry_kernel(const __grid_constant__ RecurP p, float* __restrict__ U,
                                                        const float* __restrict__ decay, int chunks, int pos0) {
  pdl_wait();
  pdl_launch_dependents();
  constexpr int W = sizeof(V) / 4;
  const int i = (blockIdx.x * 256 + threadIdx.x) * W, n = p.H * p.D * p.E;
  if (i >= n) return;
  const int hd = i / p.E, HD = p.H * p.D;
  V s{};
  if (pos0 > 0) s = *(const V*)(p.S + i);
  for (int c0 = 0; c0 < chunks; c0 += GA_BATCH) {
    V u[GA_BATCH];
    float g[GA_BATCH];
#pragma unroll
    for (int c = 0; c < GA_BATCH; c++)
      if (c0 + c < chunks) {
        u[c] = *(const V*)(U + (size_t)(c0 + c) * n + i);
        g[c] = decay[(size_t)(c0 + c) * HD + hd];
      }
#pragma unroll
    for (int c = 0; c < GA_BATCH; c++)
      if (c0 + c < chunks) {
        *(V*)(U + (size_t)(c0 + c) * n + i) = s;
        s = fma_state(s, g[c], u[c]);
      }
  }
  *(V*)(p.S + i) = s;
}

// ---- the chunk's outputs --------------------------------------------------------------------------------
template <int DP>
struct GoSmem {
  static constexpr int LD = DP + 8;
  static constexpr size_t Q = 0;                                        // [2 planes][64][LD]
  static constexpr size_t K = Q + (size_t)2 * GC_L * LD * 2;            // the same; or b [64][DP + 1] f32; then
  static constexpr size_t KB = (size_t)2 * GC_L * LD * 2;               //   the state's planes [2][DP][GC_ELD]
  static constexpr size_t SB = (size_t)2 * DP * GC_ELD * 2;
  static constexpr size_t V = K + (KB > SB ? KB : SB);                  // [64][GC_ELD]
  static constexpr size_t G = V + (size_t)GC_L * GC_ELD * 2;            // [groups][DP] f32
  static constexpr size_t TOTAL = G + (size_t)GC_THREADS * 4;
};
template <int DP>
__global__ void __launch_bounds__(GC_THREADS, DP <= 128 ? 2 : 1)
    gla_out_kernel(const __grid_constant__ RecurP p, const float* __restrict__ proj, long long ld,
                   const float* __restrict__ rates, const float* __restrict__ U, float* __restrict__ o, int rows) {
  using SM = GoSmem<DP>;
  using B = __nv_bfloat16;
  constexpr int LD = SM::LD, NG = GC_THREADS / DP, TG = GC_L / NG;
  extern __shared__ __align__(16) unsigned char smem[];
  B* qs = (B*)(smem + SM::Q);
  B* ks = (B*)(smem + SM::K);
  float* bs = (float*)(smem + SM::K);
  B* ss = (B*)(smem + SM::K);
  B* vs = (B*)(smem + SM::V);
  float* gsum = (float*)(smem + SM::G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = p.D, E = p.E;
  const int h = blockIdx.x, ch = blockIdx.y, t0 = ch * GC_L, n = rows - t0 < GC_L ? rows - t0 : GC_L;
  const int d = tid % DP, grp = tid / DP, tg = grp * TG, HD = p.H * D;
  const int rg = warp & 3, half = warp >> 2, wr = rg * 16, ra = wr + (lane >> 2), cb = (lane & 3) * 2;
  pdl_wait();
  pdl_launch_dependents();
  const float qscale = rsqrtf((float)D);
  const float* row = proj + (size_t)(t0 + tg) * ld + h * D + d;
  {
    float x[TG];
    gsum[grp * DP + d] = load_rates<TG>(rates + (size_t)(t0 + tg) * HD + h * D + d, HD, n - tg, d < D, x);
    __syncthreads();
    float b = 0.f, all = 0.f;
#pragma unroll
    for (int g = 0; g < NG; g++) {
      if (g < grp) b += gsum[g * DP + d];
      all += gsum[g * DP + d];
    }
    const bool far = __syncthreads_or(all > GC_MOST);
#pragma unroll
    for (int i = 0; i < TG; i++) {
      const bool on = d < D && tg + i < n;
      const float qv = on ? row[(size_t)i * ld + p.cq] * qscale : 0.f, kv = on && !far ? row[(size_t)i * ld + p.ck] : 0.f;
      b += x[i];
      put_planes(qs + (tg + i) * LD + d, (size_t)GC_L * LD, qv * expf(-b));
      if (far) bs[(tg + i) * (DP + 1) + d] = b;
      else put_planes(ks + (tg + i) * LD + d, (size_t)GC_L * LD, kv * expf(b));
    }
    __syncthreads();
    // A for the rows of this warp, then as operand planes
    float m[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++) m[j][0] = m[j][1] = m[j][2] = m[j][3] = 0.f;
    if (!far) {
#pragma unroll 2
      for (int k = 0; k < DP; k += 16) {
        uint32_t ah[4], al[4];
        rc_ldm(ah, rc_a(qs, LD, wr, k, lane));
        rc_ldm(al, rc_a(qs + GC_L * LD, LD, wr, k, lane));
#pragma unroll
        for (int j = 0; j < 4; j++)
          if (j <= rg) {
            uint32_t bh[4], bl[4];
            rc_ldm(bh, rc_bn(ks, LD, j * 16, k, lane));
            rc_ldm(bl, rc_bn(ks + GC_L * LD, LD, j * 16, k, lane));
            rc_mma(m[2 * j], ah, bh[0], bh[1]); rc_mma(m[2 * j + 1], ah, bh[2], bh[3]);
            rc_mma(m[2 * j], al, bh[0], bh[1]); rc_mma(m[2 * j + 1], al, bh[2], bh[3]);
            rc_mma(m[2 * j], ah, bl[0], bl[1]); rc_mma(m[2 * j + 1], ah, bl[2], bl[3]);
          }
      }
    } else {
      const float* q0 = proj + (size_t)t0 * ld + p.cq + h * D;
      const float* k0 = proj + (size_t)t0 * ld + p.ck + h * D;
#pragma unroll
      for (int j = 0; j < 8; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const int t = ra + (e >> 1) * 8, s = j * 8 + cb + (e & 1);
          if (s <= t && t < n) {
            float a = 0.f;
            for (int c = 0; c < D; c++)
              a = fmaf(q0[(size_t)t * ld + c] * k0[(size_t)s * ld + c], expf(bs[s * (DP + 1) + c] - bs[t * (DP + 1) + c]), a);
            m[j][e] = a * qscale;
          }
        }
    }
    uint32_t mh[4][4], ml[4][4];
#pragma unroll
    for (int j = 0; j < 8; j++) {
      float w[4];
#pragma unroll
      for (int e = 0; e < 4; e++) w[e] = j * 8 + cb + (e & 1) <= ra + (e >> 1) * 8 ? m[j][e] : 0.f;
      rc_split(w[0], w[1], mh[j >> 1][(j & 1) * 2], ml[j >> 1][(j & 1) * 2]);
      rc_split(w[2], w[3], mh[j >> 1][(j & 1) * 2 + 1], ml[j >> 1][(j & 1) * 2 + 1]);
    }
    const float* S = U + ((size_t)ch * p.H + h) * D * E;
    for (int e0 = 0; e0 < E; e0 += GC_E) {
      __syncthreads();   // keys, or the columns before, are read
      load_values<GC_E>(vs, proj + (size_t)t0 * ld + p.cvv + h * E + e0, ld, n, E - e0, (E & 3) == 0);
#pragma unroll 8
      for (int i = tid; i < DP * GC_E / 2; i += GC_THREADS) {
        const int r = i / (GC_E / 2), c = (i - r * (GC_E / 2)) * 2;
        const float* at = S + (size_t)r * E + e0 + c;
        float2 v = make_float2(0.f, 0.f);
        if ((E & 1) == 0) {
          if (r < D && e0 + c < E) v = *(const float2*)at;
        } else {
          if (r < D && e0 + c < E) v.x = at[0];
          if (r < D && e0 + c + 1 < E) v.y = at[1];
        }
        uint32_t hi, lo;
        rc_split(v.x, v.y, hi, lo);
        *(uint32_t*)(ss + r * GC_ELD + c) = hi;
        *(uint32_t*)(ss + (DP + r) * GC_ELD + c) = lo;
      }
      __syncthreads();
      float y[4][4];
#pragma unroll
      for (int j = 0; j < 4; j++) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
#pragma unroll 4
      for (int k = 0; k < DP; k += 16) {
        uint32_t ah[4], al[4];
        rc_ldm(ah, rc_a(qs, LD, wr, k, lane));
        rc_ldm(al, rc_a(qs + GC_L * LD, LD, wr, k, lane));
#pragma unroll
        for (int j = 0; j < 2; j++) {
          uint32_t bh[4], bl[4];
          rc_ldmt(bh, rc_bk(ss, GC_ELD, k, half * 32 + j * 16, lane));
          rc_ldmt(bl, rc_bk(ss + DP * GC_ELD, GC_ELD, k, half * 32 + j * 16, lane));
          rc_mma(y[2 * j], ah, bh[0], bh[1]); rc_mma(y[2 * j + 1], ah, bh[2], bh[3]);
          rc_mma(y[2 * j], al, bh[0], bh[1]); rc_mma(y[2 * j + 1], al, bh[2], bh[3]);
          rc_mma(y[2 * j], ah, bl[0], bl[1]); rc_mma(y[2 * j + 1], ah, bl[2], bl[3]);
        }
      }
#pragma unroll
      for (int k = 0; k < 4; k++)
        if (k <= rg) {
#pragma unroll
          for (int j = 0; j < 2; j++) {
            uint32_t bv[4];
            rc_ldmt(bv, rc_bk(vs, GC_ELD, k * 16, half * 32 + j * 16, lane));
            rc_mma(y[2 * j], mh[k], bv[0], bv[1]); rc_mma(y[2 * j + 1], mh[k], bv[2], bv[3]);
            rc_mma(y[2 * j], ml[k], bv[0], bv[1]); rc_mma(y[2 * j + 1], ml[k], bv[2], bv[3]);
          }
        }
#pragma unroll
      for (int f = 0; f < 2; f++) {
        const int t = ra + 8 * f;
        if (t >= n) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
          const int e = e0 + half * 32 + j * 8 + cb;
          float* dst = o + ((size_t)(t0 + t) * p.H + h) * E + e;
          if ((E & 1) == 0) {
            if (e < E) *(float2*)dst = make_float2(y[j][2 * f], y[j][2 * f + 1]);
          } else {
            if (e < E) dst[0] = y[j][2 * f];
            if (e + 1 < E) dst[1] = y[j][2 * f + 1];
          }
        }
      }
    }
  }
}

template <int DP>
int gla_t(const RecurP& p, const float* proj, long long ld, const float* rates, float* U, float* decay, float* o, int rows,
          int pos0, cudaStream_t s) {
  const int chunks = (rows + GC_L - 1) / GC_L;
  constexpr int SE = GS_E<DP>;
  constexpr int sm1 = (2 * GC_L * (DP + 8) + GC_L * (SE + 8)) * 2 + GC_THREADS * 4, sm2 = (int)GoSmem<DP>::TOTAL;
  static std::atomic<unsigned long long> d1{0}, d2{0};
  int rc = ensure_dynamic_smem(gla_state_kernel<DP>, sm1, d1);
  if (!rc) rc = ensure_dynamic_smem(gla_out_kernel<DP>, sm2, d2);
  if (rc) return rc;
  LaunchCfg l1(dim3((p.E + SE - 1) / SE, p.H, chunks), dim3(GC_THREADS), sm1, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&l1.cfg, gla_state_kernel<DP>, p, proj, ld, rates, U, decay, rows));
  const int w = (p.E & 3) == 0 ? 4 : 1;
  LaunchCfg l2(dim3((p.H * p.D * p.E / w + 255) / 256), dim3(256), 0, s, pdl_enabled());
  if (w == 4) TLB_CUDA(cudaLaunchKernelEx(&l2.cfg, gla_carry_kernel<float4>, p, U, (const float*)decay, chunks, pos0));
  else TLB_CUDA(cudaLaunchKernelEx(&l2.cfg, gla_carry_kernel<float>, p, U, (const float*)decay, chunks, pos0));
  LaunchCfg l3(dim3(p.H, chunks), dim3(GC_THREADS), sm2, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&l3.cfg, gla_out_kernel<DP>, p, proj, ld, rates, (const float*)U, o, rows));
  return TLB_OK;
}

}  // namespace

int gla_rates_launch(const RecurP& p, const float* proj, long long ld, float* rates, int rows, cudaStream_t s) {
  LaunchCfg lc(dim3((p.H * p.D + 255) / 256, (rows + GR_ROWS - 1) / GR_ROWS), dim3(256), 0, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, gla_rates_kernel, p, proj, ld, rates, rows));
  return TLB_OK;
}

bool gla_chunk_eligible(const RecurP& p) { return p.D <= 256; }

static size_t gla_u_floats(const RecurP& p, int rows) {
  return ((size_t)((rows + GC_L - 1) / GC_L) * p.H * p.D * p.E + 3) & ~(size_t)3;
}
size_t gla_chunk_scratch_bytes(const RecurP& p, int rows) {
  return (gla_u_floats(p, rows) + (size_t)((rows + GC_L - 1) / GC_L) * p.H * p.D) * sizeof(float);
}

int gla_chunk_launch(const RecurP& p, const float* proj, long long ld, const float* rates, void* scratch, float* o,
                     int rows, int pos0, cudaStream_t s) {
  float *U = (float*)scratch, *decay = U + gla_u_floats(p, rows);
  if (p.D <= 64) return gla_t<64>(p, proj, ld, rates, U, decay, o, rows, pos0, s);
  if (p.D <= 128) return gla_t<128>(p, proj, ld, rates, U, decay, o, rows, pos0, s);
  return gla_t<256>(p, proj, ld, rates, U, decay, o, rows, pos0, s);
}

}  // namespace tlb
