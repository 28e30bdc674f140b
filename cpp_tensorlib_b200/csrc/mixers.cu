// Sequence mixers of the layer-stack decoder (see mixers.cuh for what each one computes).
//
// One token: ONE launch for all mixers of a layer.  Blocks are divided among them by index: the
// attention takes (key/value head, head block, key range) units whose last arriver merges the
// ranges and applies the output gate; a recurrent mixer takes one block per head, which runs the
// convolutions, the state update and the read-out, and finishes the head -- except gla, which has no
// convolution and takes a block per 32 state columns (norm and gate follow with the output projection).
// Latent attention has launches of its own (attn_latent.cu).
//
// Prompt pass: row-batched launches.  attn_rows_prep (norm, rotation, cache rows), attn_rows
// (attention of every row), recur_rows_conv (convolutions, unit norms, step sizes and decay rates),
// recur_rows_scan (the recurrence, state in registers), recur_rows_finish (norms and gates).  bf16
// models take attn_window.cu and recur_chunk.cu for attention and recurrence where the widths allow.
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
// Everything but the projected row was written at least two launches ago, and the launch before this
// one starts its successors only behind its own wait: the position, the caches, the states and the
// weights may be read before pdl_wait.
struct AttnUnit {
  int g, gb, h0, nh, split, active, t0, t1;
  Visible vis;
};
__device__ __forceinline__ AttnUnit attn_unit_of(const AttnP& p, int unit, int pos) {
  AttnUnit a;
  a.split = unit % p.splits;
  a.gb = unit / p.splits;
  a.g = a.gb / p.hb;
  a.h0 = a.g * (p.H / p.G) + (a.gb % p.hb) * p.hpb;
  const int left = (a.g + 1) * (p.H / p.G) - a.h0;
  a.nh = left < p.hpb ? left : p.hpb;
  a.vis = visible_of(p, pos);
  int chunk = (a.vis.n + p.splits - 1) / p.splits;
  chunk = chunk < 64 ? 64 : chunk;
  a.active = (a.vis.n + chunk - 1) / chunk;
  a.t0 = a.split * chunk;
  a.t1 = a.t0 + chunk < a.vis.n ? a.t0 + chunk : a.vis.n;
  return a;
}
// sum of squares of n values of the projected row, this thread's share, 16 values in flight
__device__ __forceinline__ float row_squares(const float* x, int n) {
  float s = 0.f;
  if ((n & 3) == 0) {
    for (int i = threadIdx.x * 4; i < n; i += 16 * MX_THREADS) {
      float4 v[4];
#pragma unroll
      for (int k = 0; k < 4; k++)
        v[k] = i + k * 4 * MX_THREADS < n ? *(const float4*)(x + i + k * 4 * MX_THREADS) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int k = 0; k < 4; k++) s = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, s))));
    }
  } else {
    for (int i = threadIdx.x; i < n; i += MX_THREADS) s = fmaf(x[i], x[i], s);
  }
  return s;
}
// norm weights of the unit's heads, before the projected row is there: wn [RM][Dp] | [Dp]
template <int RM>
__device__ void attn_norm_weights(const AttnP& p, const AttnUnit& a, float* wn) {
  for (int i = threadIdx.x; i < (RM + 1) * p.Dp; i += MX_THREADS) {
    const int r = i / p.Dp, d = i - r * p.Dp;
    float v = 0.f;
    if (d < p.D && r < a.nh) v = p.qn[(a.h0 + r) * p.D + d];
    if (d < p.D && r == RM) v = p.kn[a.g * p.D + d];
    wn[i] = v;
  }
}
// normed and rotated query heads of the unit into qs [RM][Dp]; with the range that ends with the token
// itself, its key and value into the cache and (in the cache's type) into knew [Dp] | [Ep]
template <typename KT, int RM>
__device__ void attn_token_heads(const AttnP& p, const AttnUnit& a, const float* row, int pos, const float2* cs,
                                 const float* wn, float* qs, KT* knew, float* red) {
  const int tid = threadIdx.x;
  const bool last = a.split == a.active - 1;
  float sq = row_squares(row + p.oq, p.H * p.D);
  float sk = last ? row_squares(row + p.ok, p.G * p.D) : 0.f;
  sq = block_sum(sq, red);
  const float rq = rsqrtf(sq / (p.H * p.D) + p.eps);
  for (int i = tid; i < RM * p.Dp; i += MX_THREADS) {
    const int r = i / p.Dp, d = i - r * p.Dp;
    float v = 0.f;
    if (r < a.nh && d < p.D) v = rot_elem(p, row + p.oq + (a.h0 + r) * p.D, wn + r * p.Dp, rq, cs, d);
    if (sizeof(KT) == 2) v = __bfloat162float(__float2bfloat16_rn(v));
    qs[i] = v;
  }
  if (last) {
    sk = block_sum(sk, red);
    const float rk = rsqrtf(sk / (p.G * p.D) + p.eps);
    const size_t slot = kv_slot(p, pos);
    KT* kd = (KT*)p.K + ((size_t)a.g * p.cap + slot) * p.Dp;
    KT* vd = (KT*)p.V + ((size_t)a.g * p.cap + slot) * p.Ep;
    for (int d = tid; d < p.Dp; d += MX_THREADS) {
      const float v = d < p.D ? rot_elem(p, row + p.ok + a.g * p.D, wn + RM * p.Dp, rk, cs, d) : 0.f;
      put(kd + d, v);
      put(knew + d, v);
    }
    for (int e = tid; e < p.Ep; e += MX_THREADS) {
      const float v = e < p.E ? row[p.ov + a.g * p.E + e] : 0.f;
      put(vd + e, v);
      put(knew + p.Dp + e, v);
    }
  }
  __syncthreads();
}

// A range's unnormalised heads (os), maxima and sums (ml) into the partials; the last range to arrive
// merges them all and applies the output gate.  Partials of a unit: [splits][hpb][Ep], then
// [splits][hpb] (maximum, sum).
template <int RM>
__device__ void attn_merge(const AttnP& p, const AttnUnit& a, float* os, float* ml, float* sc, const float* row,
                           float* out) {
  __shared__ int s_last;
  const int tid = threadIdx.x, nh = a.nh, active = a.active;
  constexpr int GH = 4;
  float gate[GH];   // of the first GH elements this thread finishes
#pragma unroll
  for (int k = 0; k < GH; k++) {
    const int i = tid + k * MX_THREADS;
    gate[k] = i < nh * p.E ? row[p.og + a.h0 * p.E + i] : 0.f;
  }
  if (active > 1) {
    const int slots = p.splits * p.hpb;
    float* part = p.part + (size_t)a.gb * attn_part_floats(p);
    float2* stat = (float2*)(part + (size_t)slots * p.Ep);
    for (int i = tid; i < nh * p.Ep / 4; i += MX_THREADS)
      ((float4*)(part + (size_t)a.split * p.hpb * p.Ep))[i] = ((const float4*)os)[i];
    if (tid < nh) stat[a.split * p.hpb + tid] = make_float2(ml[tid], ml[RM + tid]);
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(&p.counters[a.gb], 1) == active - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (tid == 0) p.counters[a.gb] = 0;
    const int warp = tid >> 5, lane = tid & 31;
    for (int r = warp; r < nh; r += MX_THREADS / 32) {
      float m = -3.0e38f;
      for (int s = lane; s < active; s += 32) m = fmaxf(m, __ldcg(&stat[s * p.hpb + r]).x);
      m = warp_max(m);
      float l = 0.f;
      for (int s = lane; s < active; s += 32) {
        const float2 v = __ldcg(&stat[s * p.hpb + r]);
        const float w = expf(v.x - m);
        sc[r * MX_TK + s] = w;
        l = fmaf(w, v.y, l);
      }
      l = warp_sum(l);
      if (lane == 0) ml[RM + r] = l;
    }
    __syncthreads();
    for (int i = tid; i < nh * p.Ep / 4; i += MX_THREADS) {
      const int r = i * 4 / p.Ep;
      const float4* src = (const float4*)part + i;
      const size_t step = (size_t)p.hpb * p.Ep / 4;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s0 = 0; s0 < active; s0 += 12) {
        float4 v[12];
#pragma unroll
        for (int k = 0; k < 12; k++)
          v[k] = s0 + k < active ? __ldcg(src + (size_t)(s0 + k) * step) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int k = 0; k < 12; k++) {
          const float w = s0 + k < active ? sc[r * MX_TK + s0 + k] : 0.f;
          acc.x = fmaf(w, v[k].x, acc.x); acc.y = fmaf(w, v[k].y, acc.y);
          acc.z = fmaf(w, v[k].z, acc.z); acc.w = fmaf(w, v[k].w, acc.w);
        }
      }
      ((float4*)os)[i] = acc;
    }
    __syncthreads();
  }
  for (int i = tid, k = 0; i < nh * p.E; i += MX_THREADS, k++) {
    const int r = i / p.E, e = i - r * p.E, c = a.h0 * p.E + i;
    float g = k == 0 ? gate[0] : (k == 1 ? gate[1] : (k == 2 ? gate[2] : gate[3]));
    if (k >= GH) g = row[p.og + c];
    out[p.oa + c] = os[r * p.Ep + e] / ml[RM + r] * sigmoid_f(g) * p.out_scale;
  }
}

// any widths, either cache type
template <typename KT, int RM>
__device__ void attn_decode_unit(const AttnP& p, int unit, const float* row, float* out, int pos, float* sm) {
  __shared__ float2 cs[MX_PAIRS];
  float* qs = sm;                         // [RM][Dp]
  float* os = qs + RM * p.Dp;             // [RM][Ep]
  float* sc = os + RM * p.Ep;             // [RM][MX_TK]
  float* ml = sc + RM * MX_TK;            // [3][RM], 32
  float* red = ml + 32;                   // [33], 40
  float* wn = red + 40;                   // [RM + 1][Dp]
  KT* knew = (KT*)(wn + (RM + 1) * p.Dp); // [Dp + Ep]
  const AttnUnit a = attn_unit_of(p, unit, pos);
  if (a.split >= a.active) { pdl_wait(); return; }
  rot_table(p, pos, cs);
  attn_norm_weights<RM>(p, a, wn);
  pdl_wait();
  pdl_launch_dependents();
  __syncthreads();
  attn_token_heads<KT, RM>(p, a, row, pos, cs, wn, qs, knew, red);
  attn_range<KT, RM>(p, qs, a.g, a.vis, a.t0, a.t1, sc, os, ml);
  attn_merge<RM>(p, a, os, ml, sc, row, out);
}

// v[N] per lane, summed over the 16 lanes of a half warp: N >= 16 leaves N / 16 sums in each lane (sum i in
// lane i % 16 of v[i / 16]), fewer leave each sum in several lanes.  Returns the index base of the lane.
template <int N>
__device__ __forceinline__ int half_warp_sums(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
  int n = N, at = 0;
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = lane & o;
#pragma unroll
      for (int i = 0; i < N / 2; i++)
        if (i < n) {
          const float send = up ? v[i] : v[i + n], keep = up ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
      if (up) at += n;
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
    }
  }
  return at;
}

// bf16 cache, widths up to 128: 64 keys a tile, 16 lanes a key row, the first tile's keys and values in
// flight before the projected row is there, and the next tile's under the current one's arithmetic
constexpr int AF_TK = 64;
template <int RM>
__device__ void attn_decode_unit16(const AttnP& p, int unit, const float* row, float* out, int pos, float* sm) {
  using KT = __nv_bfloat16;
  __shared__ float2 cs[64];
  float* qs = sm;                         // [RM][Dp]
  float* os = qs + RM * p.Dp;             // [RM][Ep]
  float* sc = os + RM * p.Ep;             // [RM][MX_TK]
  float* ml = sc + RM * MX_TK;            // [3][RM], 32
  float* red = ml + 32;                   // [33], 40
  float* wn = red + 40;                   // [RM + 1][Dp]
  KT* knew = (KT*)(wn + (RM + 1) * p.Dp); // [Dp + Ep]
  float* wo = (float*)(knew + 256);       // [8 warps][RM][Ep]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, ch = tid & 15, kr = tid >> 4;
  const AttnUnit a = attn_unit_of(p, unit, pos);
  if (a.split >= a.active) { pdl_wait(); return; }
  const KT* K = (const KT*)p.K + (size_t)a.g * p.cap * p.Dp + ch * 8;
  const KT* V = (const KT*)p.V + (size_t)a.g * p.cap * p.Ep + ch * 8;
  const bool ck = ch * 8 < p.Dp, cv = ch * 8 < p.Ep;
  uint4 kf[4], vf[4];
  auto load = [&](uint4 (&f)[4], const KT* base, int width, bool on, int tb) {
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int t = tb + kr + 16 * i;
      f[i] = make_uint4(0, 0, 0, 0);
      if (on && t < a.t1) f[i] = *(const uint4*)(base + (size_t)kv_slot(p, visible_pos(a.vis, t)) * width);
    }
  };
  load(kf, K, p.Dp, ck, a.t0);
  load(vf, V, p.Ep, cv, a.t0);
  rot_table(p, pos, cs);
  attn_norm_weights<RM>(p, a, wn);
  pdl_wait();
  pdl_launch_dependents();
  if (tid < RM) { ml[tid] = -3.0e38f; ml[RM + tid] = 0.f; }
  __syncthreads();
  attn_token_heads<KT, RM>(p, a, row, pos, cs, wn, qs, knew, red);
  float acc[RM][8];
#pragma unroll
  for (int r = 0; r < RM; r++)
#pragma unroll
    for (int e = 0; e < 8; e++) acc[r][e] = 0.f;
  for (int tb = a.t0; tb < a.t1; tb += AF_TK) {
    const int n = a.t1 - tb < AF_TK ? a.t1 - tb : AF_TK, own = a.vis.n - 1 - tb;   // place of the token itself
#pragma unroll
    for (int i = 0; i < 4; i++)
      if (kr + 16 * i == own) {
        if (ck) kf[i] = *(const uint4*)(knew + ch * 8);
        if (cv) vf[i] = *(const uint4*)(knew + p.Dp + ch * 8);
      }
    float s[4 * RM];
#pragma unroll
    for (int i = 0; i < 4; i++) {
      float f[8];
      widen16(kf[i], f, (const KT*)nullptr);
#pragma unroll
      for (int r = 0; r < RM; r++) {
        float d = 0.f;
        if (ck) {
          const float4 x = *(const float4*)(qs + r * p.Dp + ch * 8), y = *(const float4*)(qs + r * p.Dp + ch * 8 + 4);
          d = fmaf(f[0], x.x, fmaf(f[1], x.y, fmaf(f[2], x.z, f[3] * x.w)));
          d = fmaf(f[4], y.x, fmaf(f[5], y.y, fmaf(f[6], y.z, fmaf(f[7], y.w, d))));
        }
        s[i * RM + r] = d;
      }
    }
    if (tb + AF_TK < a.t1) load(kf, K, p.Dp, ck, tb + AF_TK);
    const int at = half_warp_sums<4 * RM>(s);
    constexpr int NS = 4 * RM > 16 ? 4 * RM / 16 : 1;
#pragma unroll
    for (int j = 0; j < NS; j++) {
      const int x = at + j, i = x / RM, r = x - i * RM;
      sc[r * AF_TK + kr + 16 * i] = kr + 16 * i < n ? s[j] * p.scale : -INFINITY;
    }
    __syncthreads();
    for (int r = warp; r < RM; r += MX_THREADS / 32) {
      const float x0 = sc[r * AF_TK + lane], x1 = sc[r * AF_TK + lane + 32], old = ml[r];
      const float m = warp_max(fmaxf(old, fmaxf(x0, x1)));
      const float e0 = expf(x0 - m), e1 = expf(x1 - m);
      sc[r * AF_TK + lane] = e0;
      sc[r * AF_TK + lane + 32] = e1;
      const float l = warp_sum(e0 + e1);
      if (lane == 0) {
        const float c = expf(old - m);
        ml[2 * RM + r] = c; ml[r] = m; ml[RM + r] = ml[RM + r] * c + l;
      }
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < RM; r++) {
      const float c = ml[2 * RM + r];
#pragma unroll
      for (int e = 0; e < 8; e++) acc[r][e] *= c;
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
      float f[8];
      widen16(vf[i], f, (const KT*)nullptr);
#pragma unroll
      for (int r = 0; r < RM; r++) {
        const float w = sc[r * AF_TK + kr + 16 * i];
#pragma unroll
        for (int e = 0; e < 8; e++) acc[r][e] = fmaf(w, f[e], acc[r][e]);
      }
    }
    if (tb + AF_TK < a.t1) {
      load(vf, V, p.Ep, cv, tb + AF_TK);
      __syncthreads();   // the weights are read: the next tile's scores may overwrite them
    }
  }
#pragma unroll
  for (int r = 0; r < RM; r++)
#pragma unroll
    for (int e = 0; e < 8; e++) acc[r][e] += __shfl_xor_sync(0xffffffffu, acc[r][e], 16);
  if (lane < 16 && cv)
#pragma unroll
    for (int r = 0; r < RM; r++) {
      float* d = wo + (warp * RM + r) * p.Ep + ch * 8;
      *(float4*)d = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
      *(float4*)(d + 4) = make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]);
    }
  __syncthreads();
  for (int i = tid; i < RM * p.Ep; i += MX_THREADS) {
    float x = 0.f;
#pragma unroll
    for (int w = 0; w < MX_THREADS / 32; w++) x += wo[w * RM * p.Ep + i];
    os[i] = x;
  }
  __syncthreads();
  attn_merge<RM>(p, a, os, ml, sc, row, out);
}

// ---- recurrent mixers, one token -----------------------------------------------------------
// One block a head.  A thread holds up to MX_ROWS rows of one state column, for two column blocks at a
// time; the first two blocks and the convolutions' history are fetched before the projected row is there.
__device__ void recur_decode_head(const RecurP& p, int h, const float* row, float* out, int pos, float* sm) {
  const int tid = threadIdx.x, D = p.D, E = p.E, rep = p.H / p.G, kg = h / rep, n = 2 * D + E;
  float* q = sm;               // [D]
  float* k = q + D;            // [D]
  float* v = k + D;            // [E]
  float* o = v + E;            // [E]
  float* wl = o + E;           // [n] weights of the current token
  float* red = wl + n;         // [2][MX_THREADS]
  float* rs = red + 2 * MX_THREADS;  // [33]
  float* S = p.S + (size_t)h * D * E;
  const int need = (D + MX_ROWS - 1) / MX_ROWS;
  const int VB = E < MX_THREADS / need ? E : MX_THREADS / need;
  const int RS = MX_THREADS / VB;
  const int grp = tid / VB, col = tid - grp * VB;
  const size_t stride = (size_t)RS * E;
  float s[2][MX_ROWS];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int b = 0; b < 2; b++) {
      const int e = c0 + b * VB + col;
      const int left = grp < RS && e < E && pos > 0 ? D - grp : 0;   // rows grp, grp + RS, ... below D
      const float* at = S + (size_t)grp * E + e;
#pragma unroll
      for (int i = 0; i < MX_ROWS; i++) {
        s[b][i] = i * RS < left ? *at : 0.f;
        at += stride;
      }
    }
  };
  fetch(0);
  auto channel = [&](int i) {
    return i < D ? p.cq + kg * D + i : (i < 2 * D ? p.ck + kg * D + i - D : p.cvv + h * E + i - 2 * D);
  };
  const int taps = p.cv.taps;
  const float A_log = p.A_log[h], bias = p.dt_bias[h], skip = p.kind == MIX_SSD ? p.Dskip[h] : 0.f;
  const float nw = p.kind == MIX_DELTA && tid < E ? p.norm[tid] : 0.f;
  for (int i0 = 0; i0 < n; i0 += 2 * MX_THREADS) {
    // two channels a thread, four taps at a time: every load of the history before its first use
    float y[2] = {0.f, 0.f};
    for (int a0 = 0; a0 + 1 < taps; a0 += 4) {
      float w[2][4], x[2][4];
      int at = (pos - (taps - 1 - a0) + taps) % taps;   // ring row of tap a0 (not read in front of the start)
      if (at < 0) at += taps;
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const bool on = a0 + j + 1 < taps && pos - (taps - 1 - a0 - j) >= 0;
#pragma unroll
        for (int b = 0; b < 2; b++) {
          const int i = i0 + b * MX_THREADS + tid;
          const int c = i < n ? channel(i) : 0;
          w[b][j] = on && i < n ? p.cv.w[(size_t)c * taps + a0 + j] : 0.f;
          x[b][j] = on && i < n ? p.cv.ring[(size_t)at * p.cv.C + c] : 0.f;
        }
        at = at + 1 == taps ? 0 : at + 1;
      }
#pragma unroll
      for (int j = 0; j < 4; j++) {
        y[0] = fmaf(w[0][j], x[0][j], y[0]);
        y[1] = fmaf(w[1][j], x[1][j], y[1]);
      }
    }
#pragma unroll
    for (int b = 0; b < 2; b++) {
      const int i = i0 + b * MX_THREADS + tid;
      if (i < n) {
        const int c = channel(i);
        sm[i] = p.cv.b ? y[b] + p.cv.b[c] : y[b];
        wl[i] = p.cv.w[(size_t)c * taps + taps - 1];
      }
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  const float* cur = row + p.cv.off;
  const float gate = tid < E ? row[p.og + h * E + tid] : 0.f;
  const float raw_in = row[p.ob + h], raw_step = row[p.oa_ + h];
  for (int i = tid; i < n; i += MX_THREADS) {
    const int c = channel(i);
    const float x = cur[c];
    sm[i] = silu_f(fmaf(wl[i], x, sm[i]));
    if (taps > 1 && (i >= 2 * D || h == kg * rep)) p.cv.ring[(size_t)(pos % taps) * p.cv.C + c] = x;
  }
  const bool delta = p.kind == MIX_DELTA;
  const float step = softplus_f(raw_step + bias);
  const float in = delta ? sigmoid_f(raw_in) : step, g = decay_of(expf(A_log) * step);
  __syncthreads();
  if (delta) {
    float sq = 0.f, sk = 0.f;
    for (int i = tid; i < D; i += MX_THREADS) { sq = fmaf(q[i], q[i], sq); sk = fmaf(k[i], k[i], sk); }
    sq = block_sum(sq, rs);
    sk = block_sum(sk, rs);
    const float fq = rsqrtf(sq + 1e-6f) * rsqrtf((float)D), fk = rsqrtf(sk + 1e-6f);
    for (int i = tid; i < D; i += MX_THREADS) { q[i] *= fq; k[i] *= fk; }
    __syncthreads();
  }
  for (int c0 = 0; c0 < E; c0 += 2 * VB) {
    if (c0) fetch(c0);
    float u[2], acc[2] = {0.f, 0.f};
    if (delta) {
      float dot[2] = {0.f, 0.f};
#pragma unroll
      for (int i = 0; i < MX_ROWS; i++) {
        const int r = grp + i * RS;
        const float kk = r < D ? k[r] : 0.f;
#pragma unroll
        for (int b = 0; b < 2; b++) {
          s[b][i] *= g;
          dot[b] = fmaf(kk, s[b][i], dot[b]);
        }
      }
      red[tid] = dot[0];
      red[MX_THREADS + tid] = dot[1];
      __syncthreads();
#pragma unroll
      for (int b = 0; b < 2; b++) {
        const int e = c0 + b * VB + col;
        float d = 0.f;
        for (int w = 0; w < RS; w++) d += red[b * MX_THREADS + w * VB + col];
        u[b] = grp < RS && e < E ? in * (v[e] - d) : 0.f;
      }
      __syncthreads();
    } else {
#pragma unroll
      for (int b = 0; b < 2; b++) {
        const int e = c0 + b * VB + col;
        u[b] = grp < RS && e < E ? in * v[e] : 0.f;
      }
#pragma unroll
      for (int i = 0; i < MX_ROWS; i++) { s[0][i] *= g; s[1][i] *= g; }
    }
#pragma unroll
    for (int i = 0; i < MX_ROWS; i++) {
      const int r = grp + i * RS;
      if (r < D) {
        const float kk = k[r], qq = q[r];
#pragma unroll
        for (int b = 0; b < 2; b++) {
          s[b][i] = fmaf(kk, u[b], s[b][i]);
          acc[b] = fmaf(qq, s[b][i], acc[b]);
        }
      }
    }
    red[tid] = acc[0];
    red[MX_THREADS + tid] = acc[1];
#pragma unroll
    for (int b = 0; b < 2; b++) {
      const int e = c0 + b * VB + col;
      const int left = grp < RS && e < E ? D - grp : 0;
      float* at = S + (size_t)grp * E + e;
#pragma unroll
      for (int i = 0; i < MX_ROWS; i++) {
        if (i * RS < left) *at = s[b][i];
        at += stride;
      }
    }
    __syncthreads();
    for (int i = tid; i < 2 * VB; i += MX_THREADS) {
      const int b = i / VB, c = i - b * VB, e = c0 + i;
      if (e < E) {
        float a = 0.f;
        for (int w = 0; w < RS; w++) a += red[b * MX_THREADS + w * VB + c];
        o[e] = a;
      }
    }
    __syncthreads();
  }
  if (delta) {
    float sq = 0.f;
    for (int e = tid; e < E; e += MX_THREADS) sq = fmaf(o[e], o[e], sq);
    sq = block_sum(sq, rs);
    const float r = rsqrtf(sq / E + p.eps) * p.out_scale;
    for (int e = tid; e < E; e += MX_THREADS)
      out[p.oa + h * E + e] = o[e] * r * (e == tid ? nw : p.norm[e]) * silu_f(e == tid ? gate : row[p.og + h * E + e]);
  } else {
    for (int e = tid; e < E; e += MX_THREADS)
      out[p.oa + h * E + e] = fmaf(skip, v[e], o[e]) * silu_f(e == tid ? gate : row[p.og + h * E + e]);
  }
}

// ---- gated linear attention, one token ------------------------------------------------------
// One block per (head, 32 state columns): warp w holds rows w, w + 8, ... of them.  The state and the
// decay's weights are fetched before the projected row is there.
constexpr int GL_COLS = 32, GL_WARPS = MX_THREADS / 32, GL_PRE = 16;
__device__ __forceinline__ int gla_slices(const RecurP& p) { return (p.E + GL_COLS - 1) / GL_COLS; }
__device__ void gla_decode_unit(const RecurP& p, int unit, const float* row, float* out, int pos, float* sm) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = p.D, E = p.E;
  const int nsl = gla_slices(p), h = unit / nsl, e = (unit - h * nsl) * GL_COLS + lane, HD = p.H * D;
  float* q = sm;               // [D]
  float* k = q + D;            // [D]
  float* al = k + D;           // [D]
  float* red = al + D;         // [GL_WARPS][32]
  float* S = p.S + (size_t)h * D * E + e;
  const bool on = e < E;
  float s[MX_ROWS], w[GL_PRE];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int i = 0; i < MX_ROWS; i++) {
      const int d = d0 + warp + i * GL_WARPS;
      s[i] = on && pos > 0 && d < D ? S[(size_t)d * E] : 0.f;
    }
  };
  fetch(0);
  const int c0 = h * D + tid;
#pragma unroll
  for (int r = 0; r < GL_PRE; r++) w[r] = tid < D && r < p.rank ? p.a_up[(size_t)r * HD + c0] : 0.f;
  const float b0 = tid < D ? p.a_bias[c0] : 0.f;
  pdl_wait();
  pdl_launch_dependents();
  const float v = on ? row[p.cvv + h * E + e] : 0.f;
  for (int d = tid; d < D; d += MX_THREADS) {
    const int c = h * D + d;
    q[d] = row[p.cq + c] * rsqrtf((float)D);
    k[d] = row[p.ck + c];
    float z = d == tid ? b0 : p.a_bias[c];
#pragma unroll
    for (int r = 0; r < GL_PRE; r++)
      if (r < p.rank) z = fmaf(row[p.ob + r], d == tid ? w[r] : p.a_up[(size_t)r * HD + c], z);
    for (int r = GL_PRE; r < p.rank; r++) z = fmaf(row[p.ob + r], p.a_up[(size_t)r * HD + c], z);
    al[d] = decay_of(gla_rate(z, p.tau));
  }
  __syncthreads();
  float acc = 0.f;
  for (int d0 = 0; d0 < D; d0 += GL_WARPS * MX_ROWS) {
    if (d0) fetch(d0);
#pragma unroll
    for (int i = 0; i < MX_ROWS; i++) {
      const int d = d0 + warp + i * GL_WARPS;
      if (d < D) {
        s[i] = fmaf(k[d], v, s[i] * al[d]);
        acc = fmaf(q[d], s[i], acc);
        if (on) S[(size_t)d * E] = s[i];
      }
    }
  }
  red[tid] = acc;
  __syncthreads();
  if (warp == 0 && on) {
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < GL_WARPS; i++) o += red[i * 32 + lane];
    out[p.oa + h * E + e] = o;
  }
}

__host__ __device__ inline int recur_blocks(const RecurP& p) {
  return p.kind == MIX_GLA ? p.H * ((p.E + GL_COLS - 1) / GL_COLS) : p.H;
}

template <typename KT, int RM, bool FAST>
__global__ void __launch_bounds__(MX_THREADS, 2) mixers_decode_kernel(const __grid_constant__ DecodeArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int pos = (int)*a.d_pos;
  int b = blockIdx.x;
  // recurrent heads first: they move the most bytes per block
  for (int i = 0; i < a.n_rec; i++) {
    const int n = recur_blocks(a.rec[i]);
    if (b < n) {
      if (a.rec[i].kind == MIX_GLA) gla_decode_unit(a.rec[i], b, a.proj, a.out, pos, sm);
      else recur_decode_head(a.rec[i], b, a.proj, a.out, pos, sm);
      return;
    }
    b -= n;
  }
  if (FAST) attn_decode_unit16<RM>(a.at, b, a.proj, a.out, pos, sm);
  else attn_decode_unit<KT, RM>(a.at, b, a.proj, a.out, pos, sm);
}

// ---- prompt pass: attention ----------------------------------------------------------------
template <typename KT>
__global__ void __launch_bounds__(MX_THREADS) attn_rows_prep_kernel(const __grid_constant__ AttnP p,
                                                                    const float* __restrict__ proj, long long ld,
                                                                    int pos0, KT* __restrict__ q) {
  __shared__ float red[33];
  __shared__ float2 cs[MX_PAIRS];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, pos = pos0 + t;
  const float* row = proj + (size_t)t * ld;
  rot_table(p, pos, cs);
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < p.H * p.D; i += MX_THREADS) { const float v = row[p.oq + i]; sq = fmaf(v, v, sq); }
  for (int i = tid; i < p.G * p.D; i += MX_THREADS) { const float v = row[p.ok + i]; sk = fmaf(v, v, sk); }
  sq = block_sum(sq, red);
  sk = block_sum(sk, red);
  const float rq = rsqrtf(sq / (p.H * p.D) + p.eps), rk = rsqrtf(sk / (p.G * p.D) + p.eps);
  KT* qd = q + (size_t)t * p.H * p.Dp;
  for (int i = tid; i < p.H * p.Dp; i += MX_THREADS) {
    const int h = i / p.Dp, d = i - h * p.Dp;
    put(qd + i, d < p.D ? rot_elem(p, row + p.oq + h * p.D, p.qn + h * p.D, rq, cs, d) : 0.f);
  }
  const size_t slot = kv_slot(p, pos);
  for (int i = tid; i < p.G * p.D; i += MX_THREADS) {
    const int g = i / p.D, d = i - g * p.D;
    put((KT*)p.K + ((size_t)g * p.cap + slot) * p.Dp + d,
        rot_elem(p, row + p.ok + g * p.D, p.kn + g * p.D, rk, cs, d));
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

// The same for the chunked form: a thread runs down CV_ROWS rows of two adjacent channels with the last
// inputs in registers.
constexpr int CV_ROWS = 32, CV_TAPS = 8, CV_STEP = 8;
__global__ void __launch_bounds__(256) conv_rows_kernel(const __grid_constant__ ConvP p, const float* __restrict__ proj,
                                                        long long ld, int rows, int pos0,
                                                        __nv_bfloat16* __restrict__ conv) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 2, t0 = blockIdx.y * CV_ROWS;
  if (c >= p.C) return;
  const int t1 = t0 + CV_ROWS < rows ? t0 + CV_ROWS : rows;
  const float* src = proj + p.off + c;
  float2 w[CV_TAPS], x[CV_TAPS - 1 + CV_STEP];   // x: the last inputs, then those of CV_STEP rows
#pragma unroll
  for (int a = 0; a < CV_TAPS; a++) {
    const int k = a - (CV_TAPS - p.taps), d = CV_TAPS - 1 - a, q = pos0 + t0 - d;
    w[a] = k >= 0 ? make_float2(p.w[(size_t)c * p.taps + k], p.w[(size_t)(c + 1) * p.taps + k]) : make_float2(0.f, 0.f);
    if (d == 0) continue;
    x[a] = make_float2(0.f, 0.f);
    if (k >= 0 && q >= 0)
      x[a] = d <= t0 ? *(const float2*)(src + (size_t)(t0 - d) * ld)
                     : *(const float2*)(p.ring + (size_t)(q % p.taps) * p.C + c);
  }
  const float2 b = p.b ? make_float2(p.b[c], p.b[c + 1]) : make_float2(0.f, 0.f);
  for (int t = t0; t < t1; t += CV_STEP) {
#pragma unroll
    for (int i = 0; i < CV_STEP; i++)
      x[CV_TAPS - 1 + i] = t + i < t1 ? *(const float2*)(src + (size_t)(t + i) * ld) : make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < CV_STEP; i++) {
      float2 y = b;
#pragma unroll
      for (int a = 0; a < CV_TAPS; a++) {
        y.x = fmaf(w[a].x, x[a + i].x, y.x);
        y.y = fmaf(w[a].y, x[a + i].y, y.y);
      }
      if (t + i < t1)
        *(__nv_bfloat162*)(conv + (size_t)(t + i) * p.C + c) = __floats2bfloat162_rn(silu_f(y.x), silu_f(y.y));
    }
#pragma unroll
    for (int a = 0; a + 1 < CV_TAPS; a++) x[a] = x[a + CV_STEP];
  }
}
// step sizes and rates, and for the delta rule the unit-norm factors of (query, key) groups
__global__ void __launch_bounds__(256) recur_scalars_kernel(const __grid_constant__ RecurP p,
                                                            const float* __restrict__ proj, long long ld,
                                                            const __nv_bfloat16* __restrict__ conv,
                                                            float2* __restrict__ gates, float2* __restrict__ norms) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const float* row = proj + (size_t)t * ld;
  for (int h = threadIdx.x; h < p.H; h += blockDim.x) gates[(size_t)t * p.H + h] = recur_gates(p, row, h);
  if (p.kind != MIX_DELTA) return;
  for (int g = threadIdx.x >> 5; g < p.G; g += blockDim.x >> 5) {
    const __nv_bfloat162* q = (const __nv_bfloat162*)(conv + (size_t)t * p.cv.C + p.cq + g * p.D);
    const __nv_bfloat162* k = (const __nv_bfloat162*)(conv + (size_t)t * p.cv.C + p.ck + g * p.D);
    float sq = 0.f, sk = 0.f;
    for (int i = lane; i < p.D / 2; i += 32) {
      const float2 a = __bfloat1622float2(q[i]), b = __bfloat1622float2(k[i]);
      sq = fmaf(a.x, a.x, fmaf(a.y, a.y, sq));
      sk = fmaf(b.x, b.x, fmaf(b.y, b.y, sk));
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0)
      norms[(size_t)t * p.G + g] = make_float2(rsqrtf(sq + 1e-6f) * rsqrtf((float)p.D), rsqrtf(sk + 1e-6f));
  }
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
// rows of the pass.  Rows of k, q and v (gla: and of the decays) of SC_T tokens at a time through shared
// memory.  `gates`: (step size, rate) per head, or the rates per key channel of gla.
constexpr int SC_T = 16, SC_WARPS = 4;

template <int KIND, int LPC, int RPL>
__global__ void __launch_bounds__(SC_WARPS * 32) recur_scan_kernel(const __grid_constant__ RecurP p,
                                                                   const float* __restrict__ conv, long long ld,
                                                                   const void* __restrict__ gates,
                                                                   float* __restrict__ o, int rows, int pos0) {
  constexpr bool DELTA = KIND == MIX_DELTA, GLA = KIND == MIX_GLA;
  constexpr int CPW = 32 / LPC, CPB = CPW * SC_WARPS, DR = LPC * RPL;
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                  // [SC_T][DR]
  float* qs = ks + SC_T * DR;      // [SC_T][DR]
  float* vs = qs + SC_T * DR;      // [SC_T][CPB]
  float2* gs = (float2*)(vs + SC_T * CPB);
  float* as = (float*)(gs + SC_T);  // gla: [SC_T][DR]
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
      const float* src = conv + (size_t)(tb + t) * ld;
      ks[i] = d < D ? src[p.ck + kg * D + d] : 0.f;
      qs[i] = d < D ? (GLA ? src[p.cq + kg * D + d] * rsqrtf((float)D) : src[p.cq + kg * D + d]) : 0.f;
      if (GLA) as[i] = d < D ? decay_of(((const float*)gates)[((size_t)(tb + t) * p.H + h) * D + d]) : 0.f;
    }
    for (int i = tid; i < n * CPB; i += SC_WARPS * 32) {
      const int t = i / CPB, c = i - t * CPB;
      vs[i] = c0 + c < E ? conv[(size_t)(tb + t) * ld + p.cvv + h * E + c0 + c] : 0.f;
    }
    if (!GLA && tid < n) {
      const float2 gt = ((const float2*)gates)[(size_t)(tb + tid) * p.H + h];
      gs[tid] = make_float2(gt.x, decay_of(gt.y));
    }
    __syncthreads();
    for (int t = 0; t < n; t++) {
      const float2 gt = GLA ? make_float2(0.f, 0.f) : gs[t];
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
      } else if (GLA) {
        u = v;
        const float4* a4 = (const float4*)(as + t * DR) + lr;
#pragma unroll
        for (int i = 0; i < RPL; i += 4) {
          const float4 x = a4[(i >> 2) * LPC];
          s[i] *= x.x; s[i + 1] *= x.y; s[i + 2] *= x.z; s[i + 3] *= x.w;
        }
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

__device__ __forceinline__ float4 ld4(const float* p) { return *(const float4*)p; }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 v = *(const uint2*)p;
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                     __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void st4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *(uint2*)p = make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
}
__device__ __forceinline__ float sq4(float4 v, float s) {
  return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
}

// delta rule and gla: per-head norm, gate.  One warp per (row, head).
template <typename OT>
__global__ void __launch_bounds__(256) delta_finish_kernel(const __grid_constant__ RecurP p, const float* __restrict__ o,
                                                           const float* __restrict__ proj, long long ld,
                                                           OT* __restrict__ act, long long lda) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const bool vec = (p.E & 3) == 0;
  for (int h = threadIdx.x >> 5; h < p.H; h += blockDim.x >> 5) {
    const float* src = o + ((size_t)t * p.H + h) * p.E;
    const float* gate = proj + (size_t)t * ld + p.og + h * p.E;
    OT* dst = act + (size_t)t * lda + p.oa + h * p.E;
    float sq = 0.f;
    if (vec) {
      for (int e = lane * 4; e < p.E; e += 128) sq = sq4(ld4(src + e), sq);
    } else {
      for (int e = lane; e < p.E; e += 32) sq = fmaf(src[e], src[e], sq);
    }
    const float r = rsqrtf(warp_sum(sq) / p.E + p.eps) * p.out_scale;
    if (vec) {
      for (int e = lane * 4; e < p.E; e += 128) {
        const float4 v = ld4(src + e), g = ld4(gate + e), w = ld4(p.norm + e);
        st4(dst + e, make_float4(v.x * r * w.x * silu_f(g.x), v.y * r * w.y * silu_f(g.y), v.z * r * w.z * silu_f(g.z),
                                 v.w * r * w.w * silu_f(g.w)));
      }
    } else {
      for (int e = lane; e < p.E; e += 32) put(dst + e, src[e] * r * p.norm[e] * silu_f(gate[e]));
    }
  }
}
// ssd: skip, gate, then the norm in equal parts.  One warp per (row, part); head widths and parts that
// are multiples of 4 go four at a time, the first SF_HOLD of them held in registers between the passes.
constexpr int SF_HOLD = 8;
template <typename OT, typename CT>
__global__ void __launch_bounds__(256) ssd_finish_kernel(const __grid_constant__ RecurP p, const float* __restrict__ o,
                                                         const CT* __restrict__ conv, const float* __restrict__ proj,
                                                         long long ld, OT* __restrict__ act, long long lda,
                                                         int norm_groups, int rows) {
  pdl_wait();
  pdl_launch_dependents();
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, t = u / norm_groups;
  if (t >= rows) return;
  const int n = p.H * p.E, m = n / norm_groups, i0 = (u - t * norm_groups) * m;
  const float* gate = proj + (size_t)t * ld + p.og;
  const CT* x = conv + (size_t)t * p.cv.C + p.cvv;
  const float* src = o + (size_t)t * n;
  OT* dst = act + (size_t)t * lda + p.oa;
  float sq = 0.f;
  if (((p.E | m) & 3) == 0) {
    auto y4 = [&](int i) {
      const float d = p.Dskip[i / p.E];
      const float4 a = ld4(src + i), b = ld4(x + i), g = ld4(gate + i);
      return make_float4(fmaf(d, b.x, a.x) * silu_f(g.x), fmaf(d, b.y, a.y) * silu_f(g.y), fmaf(d, b.z, a.z) * silu_f(g.z),
                         fmaf(d, b.w, a.w) * silu_f(g.w));
    };
    float4 v[SF_HOLD];
#pragma unroll
    for (int k = 0; k < SF_HOLD; k++) {
      const int i = lane * 4 + k * 128;
      v[k] = i < m ? y4(i0 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      sq = sq4(v[k], sq);
    }
    for (int i = lane * 4 + SF_HOLD * 128; i < m; i += 128) sq = sq4(y4(i0 + i), sq);
    const float r = rsqrtf(warp_sum(sq) / m + p.eps) * p.out_scale;
    auto out4 = [&](int i, float4 y) {
      const float4 w = ld4(p.norm + i);
      st4(dst + i, make_float4(y.x * r * w.x, y.y * r * w.y, y.z * r * w.z, y.w * r * w.w));
    };
#pragma unroll
    for (int k = 0; k < SF_HOLD; k++) {
      const int i = lane * 4 + k * 128;
      if (i < m) out4(i0 + i, v[k]);
    }
    for (int i = lane * 4 + SF_HOLD * 128; i < m; i += 128) out4(i0 + i, y4(i0 + i));
    return;
  }
  auto y1 = [&](int i) { return fmaf(p.Dskip[i / p.E], to_f(x[i]), src[i]) * silu_f(gate[i]); };
  for (int i = lane; i < m; i += 32) { const float y = y1(i0 + i); sq = fmaf(y, y, sq); }
  const float r = rsqrtf(warp_sum(sq) / m + p.eps) * p.out_scale;
  for (int i = lane; i < m; i += 32) put(dst + i0 + i, y1(i0 + i) * r * p.norm[i0 + i]);
}

size_t attn_smem(const AttnP& p, int rm) {
  const int fast = p.Dp <= 128 && p.Ep <= 128 ? 8 * rm * p.Ep + 128 : 0;
  return (size_t)(rm * (2 * p.Dp + p.Ep + MX_TK) + 32 + 40 + 2 * p.Dp + p.Ep + fast) * sizeof(float);
}
size_t recur_smem(const RecurP& p) {
  if (p.kind == MIX_GLA) return (size_t)(3 * p.D + MX_THREADS) * sizeof(float);
  return (size_t)(4 * p.D + 3 * p.E + 2 * MX_THREADS + 40) * sizeof(float);
}
int rm_of(int hpb) { return hpb <= 1 ? 1 : (hpb <= 2 ? 2 : (hpb <= 4 ? 4 : 8)); }

template <typename KT, int RM, bool FAST>
int decode_launch(const DecodeArgs& a, int blocks, size_t smem, cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(mixers_decode_kernel<KT, RM, FAST>, 200 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3(blocks), dim3(MX_THREADS), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, mixers_decode_kernel<KT, RM, FAST>, a));
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
template <int KIND, int LPC, int RPL>
int scan_t(const RecurP& p, const float* conv, long long ld, const void* gates, float* o, int rows, int pos0,
           cudaStream_t s) {
  constexpr int CPB = 32 / LPC * SC_WARPS, DR = LPC * RPL;
  const size_t smem = (size_t)((KIND == MIX_GLA ? 3 : 2) * SC_T * DR + SC_T * CPB + 2 * SC_T) * sizeof(float);
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(recur_scan_kernel<KIND, LPC, RPL>, 200 * 1024, done);
  if (rc) return rc;
  LaunchCfg lc(dim3((p.E + CPB - 1) / CPB, p.H), dim3(SC_WARPS * 32), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, recur_scan_kernel<KIND, LPC, RPL>, p, conv, ld, gates, o, rows, pos0));
  return TLB_OK;
}
template <int KIND>
int scan_d(const RecurP& p, const float* conv, long long ld, const void* gates, float* o, int rows, int pos0,
           cudaStream_t s) {
  if (p.D <= 32) return scan_t<KIND, 8, 4>(p, conv, ld, gates, o, rows, pos0, s);
  if (p.D <= 64) return scan_t<KIND, 8, 8>(p, conv, ld, gates, o, rows, pos0, s);
  if (p.D <= 128) return scan_t<KIND, 8, 16>(p, conv, ld, gates, o, rows, pos0, s);
  if (p.D <= 256) return scan_t<KIND, 8, 32>(p, conv, ld, gates, o, rows, pos0, s);
  if (p.D <= 1024) return scan_t<KIND, 32, 32>(p, conv, ld, gates, o, rows, pos0, s);
  return set_error(TLB_ERR_UNSUPPORTED, "recurrent mixer: state width above 1024");
}

}  // namespace

int mixers_decode_launch(const AttnP* attn, const RecurP* rec, int n_rec, const float* proj, float* out,
                         const unsigned* d_pos, bool kv_bf16, cudaStream_t s) {
  DecodeArgs a{};
  int rm = 1;
  size_t smem = 0;
  bool fast = true;
  if (attn) {
    a.at = *attn;
    fast = attn->Dp <= 128 && attn->Ep <= 128;
    a.n_attn = attn->G * attn->hb * attn->splits;
    rm = rm_of(attn->hpb);
    smem = attn_smem(*attn, rm);
  }
  a.n_rec = n_rec;
  int blocks = a.n_attn;
  for (int i = 0; i < n_rec; i++) {
    a.rec[i] = rec[i];
    blocks += recur_blocks(rec[i]);
    const size_t n = recur_smem(rec[i]);
    smem = n > smem ? n : smem;
  }
  a.proj = proj; a.out = out; a.d_pos = d_pos;
#define MX_CASE(m)                                                                     \
  if (rm == m)                                                                         \
    return !kv_bf16 ? decode_launch<float, m, false>(a, blocks, smem, s)                  \
           : fast   ? decode_launch<__nv_bfloat16, m, true>(a, blocks, smem, s)           \
                    : decode_launch<__nv_bfloat16, m, false>(a, blocks, smem, s);
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

int recur_rows_conv_launch(const RecurP& p, const float* proj, long long ld, int rows, int pos0, void* conv,
                           float2* gates, float2* norms, bool chunked, cudaStream_t s) {
  if (chunked && p.cv.taps > CV_TAPS) return set_error(TLB_ERR_UNSUPPORTED, "recurrent mixer: convolution too long");
  if (chunked) {
    LaunchCfg lc(dim3((p.cv.C / 2 + 255) / 256, (rows + CV_ROWS - 1) / CV_ROWS), dim3(256), 0, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, conv_rows_kernel, p.cv, proj, ld, rows, pos0, (__nv_bfloat16*)conv));
    LaunchCfg ls(dim3(rows), dim3(256), 0, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&ls.cfg, recur_scalars_kernel, p, proj, ld, (const __nv_bfloat16*)conv, gates, norms));
  } else {
    LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, recur_conv_kernel, p, proj, ld, pos0, (float*)conv, gates));
  }
  if (p.cv.taps > 1) {
    LaunchCfg lc(dim3((p.cv.C + 127) / 128, p.cv.taps - 1), dim3(128), 0, s, pdl_enabled());
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, conv_ring_kernel, p.cv, proj, ld, rows, pos0));
  }
  return TLB_OK;
}

int recur_rows_scan_launch(const RecurP& p, const float* conv, long long ld, const void* gates, float* o, int rows,
                           int pos0, cudaStream_t s) {
  if (p.kind == MIX_GLA) return scan_d<MIX_GLA>(p, conv, ld, gates, o, rows, pos0, s);
  return p.kind == MIX_DELTA ? scan_d<MIX_DELTA>(p, conv, ld, gates, o, rows, pos0, s)
                             : scan_d<MIX_SSD>(p, conv, ld, gates, o, rows, pos0, s);
}

int recur_rows_finish_launch(const RecurP& p, const float* o, const void* conv, bool conv_bf16, const float* proj,
                             long long ld, void* act, long long lda, int norm_groups, int rows, bool bf16, cudaStream_t s) {
  using B = __nv_bfloat16;
  if (p.kind != MIX_SSD) {
    LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
    if (bf16) TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, delta_finish_kernel<B>, p, o, proj, ld, (B*)act, lda));
    else TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, delta_finish_kernel<float>, p, o, proj, ld, (float*)act, lda));
    return TLB_OK;
  }
  LaunchCfg lc(dim3((unsigned)(((long long)rows * norm_groups + 7) / 8)), dim3(256), 0, s, pdl_enabled());
  if (bf16 && conv_bf16)
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, ssd_finish_kernel<B, B>, p, o, (const B*)conv, proj, ld, (B*)act, lda, norm_groups, rows));
  else if (bf16)
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, ssd_finish_kernel<B, float>, p, o, (const float*)conv, proj, ld, (B*)act, lda, norm_groups, rows));
  else
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, ssd_finish_kernel<float, float>, p, o, (const float*)conv, proj, ld, (float*)act, lda, norm_groups, rows));
  return TLB_OK;
}

}  // namespace tlb
