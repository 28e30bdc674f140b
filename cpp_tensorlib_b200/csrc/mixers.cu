// Sequence mixers of the layer-stack decoder (see mixers.cuh for what each one computes).
//
// One token: ONE launch for all mixers of a layer.  Blocks are divided among them by index: the
// attention takes (key/value head, head block, key range) units whose last arriver merges the
// ranges and applies the output gate; a recurrent mixer takes one block per head, which runs the
// convolutions, the state update and the read-out, and finishes the head.
//
// Prompt pass: row-batched launches.  attn_rows_prep (norm, rotation, cache rows), attn_rows
// (attention of every row), recur_rows_conv (convolutions, unit norms, step sizes and decays),
// recur_rows_scan (the recurrence, state in registers), recur_rows_finish (norms and gates).
#include "mixers.cuh"

namespace tlb {

namespace {

constexpr int MX_MAXREC = 2;
constexpr int MX_ROWS = 32;     // state rows per thread of the one-token update

struct DecodeArgs {
  AttnP at;
  RecurP rec[MX_MAXREC];
  int n_attn;                   // blocks of the attention (0: the layer has none)
  int n_rec;
  const float* proj;
  float* out;
  const unsigned* d_pos;
};

// ---- attention, one token ------------------------------------------------------------------
template <typename KT, int RM>
__device__ void attn_finish(const AttnP& p, const float* os, const float* ml, int h0, int nh, const float* row,
                            float* out) {
  for (int i = threadIdx.x; i < nh * p.E; i += MX_THREADS) {
    const int r = i / p.E, e = i - r * p.E, c = (h0 + r) * p.E + e;
    out[p.oa + c] = os[r * p.Ep + e] / ml[RM + r] * sigmoid_f(row[p.og + c]) * p.out_scale;
  }
}

template <typename KT, int RM>
__device__ void attn_decode_unit(const AttnP& p, int unit, const float* row, float* out, int pos, float* sm) {
  __shared__ int s_last;
  float* qs = sm;                         // [RM][Dp]
  float* os = qs + RM * p.Dp;             // [RM][Ep]
  float* sc = os + RM * p.Ep;             // [RM][MX_TK]
  float* ml = sc + RM * MX_TK;            // [3][RM]
  float* red = ml + 3 * RM;               // [33]
  const int tid = threadIdx.x, split = unit % p.splits, gb = unit / p.splits;
  const int g = gb / p.hb, h0 = g * (p.H / p.G) + (gb % p.hb) * p.hpb;
  const int left = (g + 1) * (p.H / p.G) - h0, nh = left < p.hpb ? left : p.hpb;
  const Visible vis = visible_of(p, pos);
  int chunk = (vis.n + p.splits - 1) / p.splits;
  chunk = chunk < 64 ? 64 : chunk;
  const int active = (vis.n + chunk - 1) / chunk;
  if (split >= active) return;
  const int t0 = split * chunk, t1 = t0 + chunk < vis.n ? t0 + chunk : vis.n;

  float sq = 0.f;
  for (int i = tid; i < p.H * p.D; i += MX_THREADS) { const float v = row[p.oq + i]; sq = fmaf(v, v, sq); }
  sq = block_sum(sq, red);
  const float rq = rsqrtf(sq / (p.H * p.D) + p.eps);
  for (int i = tid; i < RM * p.Dp; i += MX_THREADS) {
    const int r = i / p.Dp, d = i - r * p.Dp;
    float v = 0.f;
    if (r < nh && d < p.D) v = rot_elem(p, row + p.oq + (h0 + r) * p.D, p.qn + (h0 + r) * p.D, rq, pos, d);
    if (sizeof(KT) == 2) v = __bfloat162float(__float2bfloat16_rn(v));
    qs[i] = v;
  }
  if (split == active - 1) {   // this range ends with the token itself: put its key and value down first
    float sk = 0.f;
    for (int i = tid; i < p.G * p.D; i += MX_THREADS) { const float v = row[p.ok + i]; sk = fmaf(v, v, sk); }
    sk = block_sum(sk, red);
    const float rk = rsqrtf(sk / (p.G * p.D) + p.eps);
    const long long slot = kv_slot(p, pos);
    KT* kd = (KT*)p.K + ((size_t)g * p.cap + slot) * p.Dp;
    KT* vd = (KT*)p.V + ((size_t)g * p.cap + slot) * p.Ep;
    for (int d = tid; d < p.D; d += MX_THREADS)
      put(kd + d, rot_elem(p, row + p.ok + g * p.D, p.kn + g * p.D, rk, pos, d));
    for (int e = tid; e < p.E; e += MX_THREADS) put(vd + e, row[p.ov + g * p.E + e]);
  }
  __syncthreads();
  attn_range<KT, RM>(p, qs, g, vis, t0, t1, sc, os, ml);
  if (active == 1) {
    attn_finish<KT, RM>(p, os, ml, h0, nh, row, out);
    return;
  }
  const int PS = p.Ep + 2;
  float* part = p.part + (size_t)gb * p.splits * p.hpb * PS;
  for (int i = tid; i < nh * p.Ep; i += MX_THREADS)
    part[((size_t)split * p.hpb + i / p.Ep) * PS + i % p.Ep] = os[i];
  if (tid < nh) {
    part[((size_t)split * p.hpb + tid) * PS + p.Ep] = ml[tid];
    part[((size_t)split * p.hpb + tid) * PS + p.Ep + 1] = ml[RM + tid];
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) s_last = atomicAdd(&p.counters[gb], 1) == active - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  if (tid == 0) p.counters[gb] = 0;
  const int warp = tid >> 5, lane = tid & 31;
  for (int r = warp; r < nh; r += MX_THREADS / 32) {
    float m = -3.0e38f;
    for (int s = lane; s < active; s += 32) m = fmaxf(m, __ldcg(&part[((size_t)s * p.hpb + r) * PS + p.Ep]));
    m = warp_max(m);
    float l = 0.f;
    for (int s = lane; s < active; s += 32) {
      const float w = expf(__ldcg(&part[((size_t)s * p.hpb + r) * PS + p.Ep]) - m);
      sc[r * MX_TK + s] = w;
      l = fmaf(w, __ldcg(&part[((size_t)s * p.hpb + r) * PS + p.Ep + 1]), l);
    }
    l = warp_sum(l);
    if (lane == 0) ml[RM + r] = l;
  }
  __syncthreads();
  for (int i = tid; i < nh * p.Ep; i += MX_THREADS) {
    const int r = i / p.Ep, e = i - r * p.Ep;
    float a = 0.f;
    for (int s = 0; s < active; s++) a = fmaf(sc[r * MX_TK + s], __ldcg(&part[((size_t)s * p.hpb + r) * PS + e]), a);
    os[i] = a;
  }
  __syncthreads();
  attn_finish<KT, RM>(p, os, ml, h0, nh, row, out);
}

// ---- recurrent mixers, one token -----------------------------------------------------------
__device__ void recur_decode_head(const RecurP& p, int h, const float* row, float* out, int pos, float* sm) {
  const int tid = threadIdx.x, D = p.D, E = p.E, rep = p.H / p.G, kg = h / rep;
  float* q = sm;               // [D]
  float* k = q + D;            // [D]
  float* v = k + D;            // [E]
  float* o = v + E;            // [E]
  float* red = o + E;          // [MX_THREADS]
  float* rs = red + MX_THREADS;  // [33]
  const float* cur = row + p.cv.off;
  for (int i = tid; i < 2 * D + E; i += MX_THREADS) {
    const int c = i < D ? p.cq + kg * D + i : (i < 2 * D ? p.ck + kg * D + i - D : p.cvv + h * E + i - 2 * D);
    sm[i] = conv_silu(p.cv, cur, 0, 0, pos, c);
    if (p.cv.taps > 1 && (i >= 2 * D || h == kg * rep)) p.cv.ring[(size_t)(pos % p.cv.taps) * p.cv.C + c] = cur[c];
  }
  __syncthreads();
  if (p.kind == MIX_DELTA) {
    float sq = 0.f, sk = 0.f;
    for (int i = tid; i < D; i += MX_THREADS) { sq = fmaf(q[i], q[i], sq); sk = fmaf(k[i], k[i], sk); }
    sq = block_sum(sq, rs);
    sk = block_sum(sk, rs);
    const float fq = rsqrtf(sq + 1e-6f) * rsqrtf((float)D), fk = rsqrtf(sk + 1e-6f);
    for (int i = tid; i < D; i += MX_THREADS) { q[i] *= fq; k[i] *= fk; }
    __syncthreads();
  }
  const float2 gt = recur_gates(p, row, h);
  float* S = p.S + (size_t)h * D * E;
  const int need = (D + MX_ROWS - 1) / MX_ROWS;
  const int VB = E < MX_THREADS / need ? E : MX_THREADS / need;
  const int RS = MX_THREADS / VB;
  const int grp = tid / VB, col = tid - grp * VB;
  for (int c0 = 0; c0 < E; c0 += VB) {
    const int e = c0 + col;
    const bool on = grp < RS && e < E;
    float s[MX_ROWS];
    float dot = 0.f;
#pragma unroll
    for (int i = 0; i < MX_ROWS; i++) {
      const int r = grp + i * RS;
      s[i] = on && r < D && pos > 0 ? S[(size_t)r * E + e] : 0.f;
    }
    float u;
    if (p.kind == MIX_DELTA) {
#pragma unroll
      for (int i = 0; i < MX_ROWS; i++) {
        const int r = grp + i * RS;
        s[i] *= gt.y;
        if (r < D) dot = fmaf(k[r], s[i], dot);
      }
      red[tid] = dot;
      __syncthreads();
      dot = 0.f;
      if (on) for (int w = 0; w < RS; w++) dot += red[w * VB + col];
      u = on ? gt.x * (v[e] - dot) : 0.f;
      __syncthreads();
    } else {
      u = on ? gt.x * v[e] : 0.f;
#pragma unroll
      for (int i = 0; i < MX_ROWS; i++) s[i] *= gt.y;
    }
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < MX_ROWS; i++) {
      const int r = grp + i * RS;
      if (on && r < D) {
        s[i] = fmaf(k[r], u, s[i]);
        acc = fmaf(q[r], s[i], acc);
        S[(size_t)r * E + e] = s[i];
      }
    }
    red[tid] = acc;
    __syncthreads();
    if (on && grp == 0) {
      acc = 0.f;
      for (int w = 0; w < RS; w++) acc += red[w * VB + col];
      o[e] = acc;
    }
    __syncthreads();
  }
  if (p.kind == MIX_DELTA) {
    float sq = 0.f;
    for (int e = tid; e < E; e += MX_THREADS) sq = fmaf(o[e], o[e], sq);
    sq = block_sum(sq, rs);
    const float r = rsqrtf(sq / E + p.eps) * p.out_scale;
    for (int e = tid; e < E; e += MX_THREADS) out[p.oa + h * E + e] = o[e] * r * p.norm[e] * silu_f(row[p.og + h * E + e]);
  } else {
    for (int e = tid; e < E; e += MX_THREADS)
      out[p.oa + h * E + e] = fmaf(p.Dskip[h], v[e], o[e]) * silu_f(row[p.og + h * E + e]);
  }
}

template <typename KT, int RM>
__global__ void __launch_bounds__(MX_THREADS) mixers_decode_kernel(const __grid_constant__ DecodeArgs a) {
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int pos = (int)*a.d_pos;
  int b = blockIdx.x;
  // recurrent heads first: they move the most bytes per block
  for (int i = 0; i < a.n_rec; i++) {
    if (b < a.rec[i].H) {
      recur_decode_head(a.rec[i], b, a.proj, a.out, pos, sm);
      return;
    }
    b -= a.rec[i].H;
  }
  attn_decode_unit<KT, RM>(a.at, b, a.proj, a.out, pos, sm);
}

// ---- prompt pass: attention ----------------------------------------------------------------
template <typename KT>
__global__ void __launch_bounds__(MX_THREADS) attn_rows_prep_kernel(const __grid_constant__ AttnP p,
                                                                    const float* __restrict__ proj, long long ld,
                                                                    int pos0, KT* __restrict__ q) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, pos = pos0 + t;
  const float* row = proj + (size_t)t * ld;
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < p.H * p.D; i += MX_THREADS) { const float v = row[p.oq + i]; sq = fmaf(v, v, sq); }
  for (int i = tid; i < p.G * p.D; i += MX_THREADS) { const float v = row[p.ok + i]; sk = fmaf(v, v, sk); }
  sq = block_sum(sq, red);
  sk = block_sum(sk, red);
  const float rq = rsqrtf(sq / (p.H * p.D) + p.eps), rk = rsqrtf(sk / (p.G * p.D) + p.eps);
  KT* qd = q + (size_t)t * p.H * p.Dp;
  for (int i = tid; i < p.H * p.Dp; i += MX_THREADS) {
    const int h = i / p.Dp, d = i - h * p.Dp;
    put(qd + i, d < p.D ? rot_elem(p, row + p.oq + h * p.D, p.qn + h * p.D, rq, pos, d) : 0.f);
  }
  const long long slot = kv_slot(p, pos);
  for (int i = tid; i < p.G * p.D; i += MX_THREADS) {
    const int g = i / p.D, d = i - g * p.D;
    put((KT*)p.K + ((size_t)g * p.cap + slot) * p.Dp + d,
        rot_elem(p, row + p.ok + g * p.D, p.kn + g * p.D, rk, pos, d));
  }
  for (int i = tid; i < p.G * p.E; i += MX_THREADS) {
    const int g = i / p.E, e = i - g * p.E;
    put((KT*)p.V + ((size_t)g * p.cap + slot) * p.Ep + e, row[p.ov + i]);
  }
}

// One block per (row, key/value head, head block): any widths, any window.
template <typename KT, int RM>
__global__ void __launch_bounds__(MX_THREADS) attn_rows_kernel(const __grid_constant__ AttnP p,
                                                               const KT* __restrict__ q,
                                                               const float* __restrict__ proj, long long ld,
                                                               KT* __restrict__ act, long long lda, int pos0) {
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;
  float* os = qs + RM * p.Dp;
  float* sc = os + RM * p.Ep;
  float* ml = sc + RM * MX_TK;
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, gb = blockIdx.y, tid = threadIdx.x;
  const int g = gb / p.hb, h0 = g * (p.H / p.G) + (gb % p.hb) * p.hpb;
  const int left = (g + 1) * (p.H / p.G) - h0, nh = left < p.hpb ? left : p.hpb;
  for (int i = tid; i < RM * p.Dp; i += MX_THREADS)
    qs[i] = i < nh * p.Dp ? to_f(q[((size_t)t * p.H + h0) * p.Dp + i]) : 0.f;
  const Visible vis = visible_of(p, pos0 + t);
  attn_range<KT, RM>(p, qs, g, vis, 0, vis.n, sc, os, ml);
  const float* row = proj + (size_t)t * ld;
  for (int i = tid; i < nh * p.E; i += MX_THREADS) {
    const int r = i / p.E, e = i - r * p.E, c = (h0 + r) * p.E + e;
    put(act + (size_t)t * lda + p.oa + c, os[r * p.Ep + e] / ml[RM + r] * sigmoid_f(row[p.og + c]) * p.out_scale);
  }
}

// ---- prompt pass: recurrent mixers ---------------------------------------------------------
// One warp per (row, head segment): query and key groups (unit norm for the delta rule), value heads.
__global__ void __launch_bounds__(256) recur_conv_kernel(const __grid_constant__ RecurP p,
                                                         const float* __restrict__ proj, long long ld, int pos0,
                                                         float* __restrict__ conv, float2* __restrict__ gates) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31, pos = pos0 + t;
  const float* row = proj + (size_t)t * ld;
  const float* cur = row + p.cv.off;
  float* dst = conv + (size_t)t * p.cv.C;
  for (int sgm = threadIdx.x >> 5; sgm < 2 * p.G + p.H; sgm += blockDim.x >> 5) {
    const bool val = sgm >= 2 * p.G;
    const int c0 = sgm < p.G ? p.cq + sgm * p.D : (!val ? p.ck + (sgm - p.G) * p.D : p.cvv + (sgm - 2 * p.G) * p.E);
    const int n = val ? p.E : p.D;
    float sq = 0.f;
    for (int i = lane; i < n; i += 32) {
      const float y = conv_silu(p.cv, cur, ld, t, pos, c0 + i);
      dst[c0 + i] = y;
      sq = fmaf(y, y, sq);
    }
    if (p.kind == MIX_DELTA && !val) {
      float f = rsqrtf(warp_sum(sq) + 1e-6f);
      if (sgm < p.G) f *= rsqrtf((float)p.D);
      for (int i = lane; i < n; i += 32) dst[c0 + i] *= f;   // the lane's own elements
    }
  }
  for (int h = threadIdx.x; h < p.H; h += blockDim.x) gates[(size_t)t * p.H + h] = recur_gates(p, row, h);
}

// after the convolutions of a pass: its last rows become the ring
__global__ void conv_ring_kernel(const __grid_constant__ ConvP p, const float* __restrict__ proj, long long ld,
                                 int rows, int pos0) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;   // b: rows from the end
  if (c >= p.C || b >= rows) return;
  const int t = rows - 1 - b;
  p.ring[(size_t)((pos0 + t) % p.taps) * p.C + c] = proj[(size_t)t * ld + p.off + c];
}

// The recurrence of a pass: LPC lanes share one state column, RPL rows each, in registers for all
// rows of the pass.  Rows of k, q and v of SC_T tokens at a time through shared memory.
constexpr int SC_T = 16, SC_WARPS = 4;

template <bool DELTA, int LPC, int RPL>
__global__ void __launch_bounds__(SC_WARPS * 32) recur_scan_kernel(const __grid_constant__ RecurP p,
                                                                   const float* __restrict__ conv,
                                                                   const float2* __restrict__ gates,
                                                                   float* __restrict__ o, int rows, int pos0) {
  constexpr int CPW = 32 / LPC, CPB = CPW * SC_WARPS, DR = LPC * RPL;
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                  // [SC_T][DR]
  float* qs = ks + SC_T * DR;      // [SC_T][DR]
  float* vs = qs + SC_T * DR;      // [SC_T][CPB]
  float2* gs = (float2*)(vs + SC_T * CPB);
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, c0 = blockIdx.x * CPB, cl = warp * CPW + lane / LPC, e = c0 + cl, lr = lane % LPC;
  const int kg = h / (p.H / p.G), D = p.D, E = p.E;
  const bool on = e < E;
  float* S = p.S + (size_t)h * D * E;
  float s[RPL];
#pragma unroll
  for (int i = 0; i < RPL; i++) {
    const int r = ((i >> 2) * LPC + lr) * 4 + (i & 3);
    s[i] = on && r < D && pos0 > 0 ? S[(size_t)r * E + e] : 0.f;
  }
  for (int tb = 0; tb < rows; tb += SC_T) {
    const int n = rows - tb < SC_T ? rows - tb : SC_T;
    __syncthreads();
    for (int i = tid; i < n * DR; i += SC_WARPS * 32) {
      const int t = i / DR, d = i - t * DR;
      const float* src = conv + (size_t)(tb + t) * p.cv.C;
      ks[i] = d < D ? src[p.ck + kg * D + d] : 0.f;
      qs[i] = d < D ? src[p.cq + kg * D + d] : 0.f;
    }
    for (int i = tid; i < n * CPB; i += SC_WARPS * 32) {
      const int t = i / CPB, c = i - t * CPB;
      vs[i] = c0 + c < E ? conv[(size_t)(tb + t) * p.cv.C + p.cvv + h * E + c0 + c] : 0.f;
    }
    if (tid < n) gs[tid] = gates[(size_t)(tb + tid) * p.H + h];
    __syncthreads();
    for (int t = 0; t < n; t++) {
      const float2 gt = gs[t];
      const float v = vs[t * CPB + cl];
      const float4* k4 = (const float4*)(ks + t * DR) + lr;
      const float4* q4 = (const float4*)(qs + t * DR) + lr;
      float kr[RPL];
      float u;
#pragma unroll
      for (int i = 0; i < RPL; i += 4) {
        const float4 x = k4[(i >> 2) * LPC];
        kr[i] = x.x; kr[i + 1] = x.y; kr[i + 2] = x.z; kr[i + 3] = x.w;
      }
      if (DELTA) {
        float d0 = 0.f, d1 = 0.f;
#pragma unroll
        for (int i = 0; i < RPL; i += 2) {
          s[i] *= gt.y; s[i + 1] *= gt.y;
          d0 = fmaf(kr[i], s[i], d0); d1 = fmaf(kr[i + 1], s[i + 1], d1);
        }
        d0 += d1;
#pragma unroll
        for (int w = LPC / 2; w > 0; w >>= 1) d0 += __shfl_xor_sync(0xffffffffu, d0, w);
        u = gt.x * (v - d0);
      } else {
        u = gt.x * v;
#pragma unroll
        for (int i = 0; i < RPL; i++) s[i] *= gt.y;
      }
      float a0 = 0.f, a1 = 0.f;
#pragma unroll
      for (int i = 0; i < RPL; i += 4) {
        const float4 x = q4[(i >> 2) * LPC];
        s[i] = fmaf(kr[i], u, s[i]); s[i + 1] = fmaf(kr[i + 1], u, s[i + 1]);
        s[i + 2] = fmaf(kr[i + 2], u, s[i + 2]); s[i + 3] = fmaf(kr[i + 3], u, s[i + 3]);
        a0 = fmaf(x.x, s[i], a0); a1 = fmaf(x.y, s[i + 1], a1);
        a0 = fmaf(x.z, s[i + 2], a0); a1 = fmaf(x.w, s[i + 3], a1);
      }
      a0 += a1;
#pragma unroll
      for (int w = LPC / 2; w > 0; w >>= 1) a0 += __shfl_xor_sync(0xffffffffu, a0, w);
      if (on && lr == 0) o[((size_t)(tb + t) * p.H + h) * E + e] = a0;
    }
  }
#pragma unroll
  for (int i = 0; i < RPL; i++) {
    const int r = ((i >> 2) * LPC + lr) * 4 + (i & 3);
    if (on && r < D) S[(size_t)r * E + e] = s[i];
  }
}

// delta rule: per-head norm, gate
template <typename OT>
__global__ void __launch_bounds__(256) delta_finish_kernel(const __grid_constant__ RecurP p, const float* __restrict__ o,
                                                           const float* __restrict__ proj, long long ld,
                                                           OT* __restrict__ act, long long lda) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  for (int h = threadIdx.x >> 5; h < p.H; h += blockDim.x >> 5) {
    const float* src = o + ((size_t)t * p.H + h) * p.E;
    const float* gate = proj + (size_t)t * ld + p.og + h * p.E;
    float sq = 0.f;
    for (int e = lane; e < p.E; e += 32) sq = fmaf(src[e], src[e], sq);
    const float r = rsqrtf(warp_sum(sq) / p.E + p.eps) * p.out_scale;
    for (int e = lane; e < p.E; e += 32)
      put(act + (size_t)t * lda + p.oa + h * p.E + e, src[e] * r * p.norm[e] * silu_f(gate[e]));
  }
}
// ssd: skip, gate, then the norm in equal parts
template <typename OT>
__global__ void __launch_bounds__(256) ssd_finish_kernel(const __grid_constant__ RecurP p, const float* __restrict__ o,
                                                         const float* __restrict__ conv, const float* __restrict__ proj,
                                                         long long ld, OT* __restrict__ act, long long lda,
                                                         int norm_groups) {
  extern __shared__ __align__(16) float ys[];   // [H * E]
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, n = p.H * p.E, m = n / norm_groups;
  const float* gate = proj + (size_t)t * ld + p.og;
  const float* x = conv + (size_t)t * p.cv.C + p.cvv;
  for (int i = tid; i < n; i += blockDim.x)
    ys[i] = fmaf(p.Dskip[i / p.E], x[i], o[(size_t)t * n + i]) * silu_f(gate[i]);
  __syncthreads();
  for (int g = 0; g < norm_groups; g++) {
    float sq = 0.f;
    for (int i = tid; i < m; i += blockDim.x) sq = fmaf(ys[g * m + i], ys[g * m + i], sq);
    sq = block_sum(sq, red);
    const float r = rsqrtf(sq / m + p.eps) * p.out_scale;
    for (int i = tid; i < m; i += blockDim.x)
      put(act + (size_t)t * lda + p.oa + g * m + i, ys[g * m + i] * r * p.norm[g * m + i]);
  }
}

size_t attn_smem(const AttnP& p, int rm) { return (size_t)(rm * (p.Dp + p.Ep + MX_TK + 3) + 40) * sizeof(float); }
size_t recur_smem(const RecurP& p) { return (size_t)(2 * p.D + 2 * p.E + MX_THREADS + 40) * sizeof(float); }
int rm_of(int hpb) { return hpb <= 1 ? 1 : (hpb <= 2 ? 2 : (hpb <= 4 ? 4 : 8)); }

template <typename KT, int RM>
int decode_launch(const DecodeArgs& a, int blocks, size_t smem, cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(mixers_decode_kernel<KT, RM>, 200 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3(blocks), dim3(MX_THREADS), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, mixers_decode_kernel<KT, RM>, a));
  return TLB_OK;
}
template <typename KT, int RM>
int attn_rows_t(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda, int rows,
                int pos0, cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(attn_rows_kernel<KT, RM>, 200 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3(rows, p.G * p.hb), dim3(MX_THREADS), attn_smem(p, RM), s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, attn_rows_kernel<KT, RM>, p, (const KT*)q, proj, ld, (KT*)act, lda, pos0));
  return TLB_OK;
}
template <bool DELTA, int LPC, int RPL>
int scan_t(const RecurP& p, const float* conv, const float2* gates, float* o, int rows, int pos0, cudaStream_t s) {
  constexpr int CPB = 32 / LPC * SC_WARPS, DR = LPC * RPL;
  const size_t smem = (size_t)(2 * SC_T * DR + SC_T * CPB + 2 * SC_T) * sizeof(float);
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(recur_scan_kernel<DELTA, LPC, RPL>, 200 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3((p.E + CPB - 1) / CPB, p.H), dim3(SC_WARPS * 32), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, recur_scan_kernel<DELTA, LPC, RPL>, p, conv, gates, o, rows, pos0));
  return TLB_OK;
}
template <bool DELTA>
int scan_d(const RecurP& p, const float* conv, const float2* gates, float* o, int rows, int pos0, cudaStream_t s) {
  if (p.D <= 32) return scan_t<DELTA, 8, 4>(p, conv, gates, o, rows, pos0, s);
  if (p.D <= 64) return scan_t<DELTA, 8, 8>(p, conv, gates, o, rows, pos0, s);
  if (p.D <= 128) return scan_t<DELTA, 8, 16>(p, conv, gates, o, rows, pos0, s);
  if (p.D <= 256) return scan_t<DELTA, 8, 32>(p, conv, gates, o, rows, pos0, s);
  if (p.D <= 1024) return scan_t<DELTA, 32, 32>(p, conv, gates, o, rows, pos0, s);
  return set_error(TLB_ERR_UNSUPPORTED, "recurrent mixer: state width above 1024");
}

}  // namespace

int mixers_decode_launch(const AttnP* attn, const RecurP* rec, int n_rec, const float* proj, float* out,
                         const unsigned* d_pos, bool kv_bf16, cudaStream_t s) {
  DecodeArgs a{};
  int rm = 1;
  size_t smem = 0;
  if (attn) {
    a.at = *attn;
    a.n_attn = attn->G * attn->hb * attn->splits;
    rm = rm_of(attn->hpb);
    smem = attn_smem(*attn, rm);
  }
  a.n_rec = n_rec;
  int blocks = a.n_attn;
  for (int i = 0; i < n_rec; i++) {
    a.rec[i] = rec[i];
    blocks += rec[i].H;
    const size_t n = recur_smem(rec[i]);
    smem = n > smem ? n : smem;
  }
  a.proj = proj; a.out = out; a.d_pos = d_pos;
#define MX_CASE(m)                                                                     \
  if (rm == m)                                                                         \
    return kv_bf16 ? decode_launch<__nv_bfloat16, m>(a, blocks, smem, s) : decode_launch<float, m>(a, blocks, smem, s);
  MX_CASE(1) MX_CASE(2) MX_CASE(4) MX_CASE(8)
#undef MX_CASE
  return set_error(TLB_ERR_STATE, "mixers: no head-block width");
}

int attn_rows_prep_launch(const AttnP& p, const float* proj, long long ld, int rows, int pos0, void* q, bool bf16,
                          cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(MX_THREADS), 0, s, pdl_enabled());
  if (bf16) TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, attn_rows_prep_kernel<__nv_bfloat16>, p, proj, ld, pos0, (__nv_bfloat16*)q));
  else TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, attn_rows_prep_kernel<float>, p, proj, ld, pos0, (float*)q));
  return TLB_OK;
}

int attn_rows_launch(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda, int rows,
                     int pos0, bool bf16, cudaStream_t s) {
  const int rm = rm_of(p.hpb);
#define MX_CASE(m)                                                                                      \
  if (rm == m)                                                                                          \
    return bf16 ? attn_rows_t<__nv_bfloat16, m>(p, q, proj, ld, act, lda, rows, pos0, s)                \
                : attn_rows_t<float, m>(p, q, proj, ld, act, lda, rows, pos0, s);
  MX_CASE(1) MX_CASE(2) MX_CASE(4) MX_CASE(8)
#undef MX_CASE
  return set_error(TLB_ERR_STATE, "attn_rows: no head-block width");
}

int recur_rows_conv_launch(const RecurP& p, const float* proj, long long ld, int rows, int pos0, float* conv,
                           float2* gates, cudaStream_t s) {
  {
    LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, recur_conv_kernel, p, proj, ld, pos0, conv, gates));
  }
  if (p.cv.taps > 1) {
    LaunchCfg lc(dim3((p.cv.C + 127) / 128, p.cv.taps - 1), dim3(128), 0, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, conv_ring_kernel, p.cv, proj, ld, rows, pos0));
  }
  return TLB_OK;
}

int recur_rows_scan_launch(const RecurP& p, const float* conv, const float2* gates, float* o, int rows, int pos0,
                           cudaStream_t s) {
  return p.kind == MIX_DELTA ? scan_d<true>(p, conv, gates, o, rows, pos0, s)
                             : scan_d<false>(p, conv, gates, o, rows, pos0, s);
}

int recur_rows_finish_launch(const RecurP& p, const float* o, const float* conv, const float* proj, long long ld,
                             void* act, long long lda, int norm_groups, int rows, int pos0, bool bf16, cudaStream_t s) {
  const size_t smem = p.kind == MIX_SSD ? (size_t)p.H * p.E * sizeof(float) : 0;
  LaunchCfg lc(dim3(rows), dim3(256), smem, s, pdl_enabled());
  if (p.kind == MIX_DELTA) {
    if (bf16) TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, delta_finish_kernel<__nv_bfloat16>, p, o, proj, ld, (__nv_bfloat16*)act, lda));
    else TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, delta_finish_kernel<float>, p, o, proj, ld, (float*)act, lda));
    return TLB_OK;
  }
  static std::atomic<unsigned long long> db{0}, df{0};
  if (bf16) {
    const int rc = ensure_dynamic_smem(ssd_finish_kernel<__nv_bfloat16>, 200 * 1024, db);
    if (rc) return rc;
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, ssd_finish_kernel<__nv_bfloat16>, p, o, conv, proj, ld, (__nv_bfloat16*)act, lda, norm_groups));
  } else {
    const int rc = ensure_dynamic_smem(ssd_finish_kernel<float>, 200 * 1024, df);
    if (rc) return rc;
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, ssd_finish_kernel<float>, p, o, conv, proj, ld, (float*)act, lda, norm_groups));
  }
  return TLB_OK;
}

}  // namespace tlb
