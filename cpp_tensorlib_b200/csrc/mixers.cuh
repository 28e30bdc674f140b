// Sequence mixers of the layer-stack decoder: parameters, and the device functions that the
// one-token launch and the prompt-pass launches share.
//
// A layer has one or two mixers that read the same normed input.  Their input projections are one
// fused matrix; each mixer finds its parts of the projected row at the offsets below, and leaves its
// finished heads in its own part of the row that the fused output projection reads.
//
//   attention   grouped heads, RMS norm over the whole query / key projection, partial interleaved
//               rotation, sliding window with the first tokens kept, sigmoid output gate
//   delta rule  short convolutions + silu, unit queries and keys, gated delta recurrence,
//               per-head RMS norm, silu output gate
//   ssd         Mamba-2: one convolution over x | B | C, scalar-decay recurrence, skip, silu gate
//               (the grouped norm behind it belongs to the output projection's input)
//   latent      attention over a low-rank latent that all heads share: queries through a latent of their
//               own, keys and values expanded per head from the kept latent beside one rotated key part,
//               optional sliding window and sigmoid output gate (attn_latent.cu)
//   gla         gated linear attention: one decay per key channel, per-head RMS norm, silu output gate
//               (the norm and the gate belong to the output projection's input; prompts: recur_gla.cu)
//
// What a sequence carries is addressed by absolute position, so nothing is cleared between
// sequences: keys and values live in kept slots plus a ring, latents in a ring, the convolutions' inputs in
// a ring of `taps` rows, and a recurrent state is read as zero at position 0.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace tlb {

enum : int { MIX_ATTN = 1, MIX_DELTA = 2, MIX_SSD = 3, MIX_LATENT = 4, MIX_GLA = 5 };

struct AttnP {
  int H, G, D, E;              // query heads, key/value heads, query/key width, value width
  int Dp, Ep;                  // cache row lengths (widths rounded up to 8)
  int Vs;                      // stride of value rows (a latent's value is a part of its key row)
  int window, keep, pairs;     // pairs = rotated dimensions / 2
  int oq, ok, ov, og;          // parts of the projected row
  int oa;                      // part of the finished row
  int cap, ring;               // cache rows per head = kept slots + ring
  float scale, eps, out_scale;
  const float *qn, *kn;
  const float2* inv_freq;      // [pairs] angular frequencies, high and low parts
  void *K, *V;                 // [G][cap][Dp], [G][cap][Ep]
  int splits, hb, hpb;         // key ranges of a token, head blocks of a group, heads per block
  float* part;                 // [G*hb] x ([splits][hpb][Ep] | [splits][hpb] (max, sum))
  int* counters;               // [G*hb]
};

// floats of one unit's partials (a multiple of 4: units start on 16 bytes)
__host__ __device__ inline size_t attn_part_floats(const AttnP& p) {
  return ((size_t)p.splits * p.hpb * (p.Ep + 2) + 3) & ~(size_t)3;
}

struct LatentP {
  int H, D, R, E, Q, C;        // heads; unrotated, rotated and value width; query and key/value rank
  int Dp, Rp, Ep, Qp, Cp;      // the same rounded up to 8
  int window, ring;            // visible positions; kept rows
  int oq, oc, og, oa;          // query latent, latent (rotated part behind it at oc + Cp), gate (-1: none),
                               // part of the finished row
  bool owner;                  // keeps rows of its own
  float scale, eps, out_scale;
  const float *qn, *cn;        // norms of the two latents
  const float2* inv_freq;      // [R / 2]
  const void *uq, *ukv;        // [H * (Dp + Rp)][Qp]; [H * Dp + H * Ep][Cp]
  void* rows;                  // [ring][Cp + Rp]: latent | rotated key part
  int splits;                  // most key ranges of a position
  __host__ __device__ int row() const { return Cp + Rp; }
  __host__ __device__ int qw() const { return Dp + Rp; }    // of a query head
};

struct ConvP {
  const float *w, *b;          // [C][taps], [C] or NULL
  float* ring;                 // [taps][C]: the row of position p sits at p % taps
  int C, taps, off;            // channels (padded), part of the projected row
};

struct RecurP {
  int kind;                    // MIX_DELTA / MIX_SSD / MIX_GLA
  int H, G, D, E;              // heads, key groups, key (state) width, value width
  ConvP cv;
  int cq, ck, cvv;             // channel of the first query (C), key (B) and value (x)
  int og, ob, oa_;             // gate (z), b (dt, decay input) and a parts of the projected row
  int oa;                      // part of the finished row
  float eps, out_scale;
  const float *A_log, *dt_bias, *Dskip, *norm;
  float* S;                    // [H][D][E]
  int rank;                    // gla: decay input; cq, ck, cvv are parts of the projected row
  float tau;
  const float *a_up, *a_bias;  // [rank][H * D], [H * D]
};

#ifdef __CUDACC__

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// clipped gated unit: g = min(gate, limit), u = clamp(up, -limit, limit); g sigmoid(1.702 g) (u + 1)
__device__ __forceinline__ float glu_clipped(float gate, float up, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.0f);
}
__device__ __forceinline__ float relu2(float z) { const float r = fmaxf(z, 0.f); return r * r; }

// The same value in every thread of the block; sm holds 33 floats.  Barriers inside.
__device__ __forceinline__ float block_sum(float v, float* sm) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) sm[threadIdx.x >> 5] = v;
  __syncthreads();
  if (threadIdx.x < 32) {
    float t = threadIdx.x < (blockDim.x >> 5) ? sm[threadIdx.x] : 0.f;
    t = warp_sum(t);
    if (threadIdx.x == 0) sm[32] = t;
  }
  __syncthreads();
  return sm[32];
}

template <typename T> struct Vec16 { static constexpr int N = 16 / sizeof(T); };
__device__ __forceinline__ void widen16(const uint4& w, float (&f)[4], const float*) {
  f[0] = __uint_as_float(w.x); f[1] = __uint_as_float(w.y); f[2] = __uint_as_float(w.z); f[3] = __uint_as_float(w.w);
}
__device__ __forceinline__ void widen16(const uint4& w, float (&f)[8], const __nv_bfloat16*) {
  f[0] = __uint_as_float(w.x << 16); f[1] = __uint_as_float(w.x & 0xffff0000u);
  f[2] = __uint_as_float(w.y << 16); f[3] = __uint_as_float(w.y & 0xffff0000u);
  f[4] = __uint_as_float(w.z << 16); f[5] = __uint_as_float(w.z & 0xffff0000u);
  f[6] = __uint_as_float(w.w << 16); f[7] = __uint_as_float(w.w & 0xffff0000u);
}
__device__ __forceinline__ void load2(const float* p, float& a, float& b) {
  const float2 v = *(const float2*)p; a = v.x; b = v.y;
}
__device__ __forceinline__ void load2(const __nv_bfloat16* p, float& a, float& b) {
  const uint32_t v = *(const uint32_t*)p; a = __uint_as_float(v << 16); b = __uint_as_float(v & 0xffff0000u);
}
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// cache row of position j: the kept first positions have slots of their own
__device__ __forceinline__ int kv_slot(const AttnP& p, int j) {
  return j < p.keep ? j : p.keep + (int)((unsigned)(j - p.keep) % (unsigned)p.ring);
}
// What the query at `pos` sees: `kept` first positions, then [lo, pos].
struct Visible { int kept, lo, n; };
__device__ __forceinline__ Visible visible_of(const AttnP& p, int pos) {
  Visible v;
  v.lo = pos + 1 > p.window ? pos + 1 - p.window : 0;
  v.kept = p.keep < v.lo ? p.keep : v.lo;
  v.n = v.kept + pos + 1 - v.lo;
  return v;
}
__device__ __forceinline__ int visible_pos(const Visible& v, int t) { return t < v.kept ? t : v.lo + (t - v.kept); }

// sine and cosine of pos * f.  The rounding of an f32 product grows with the position (one part in
// 2^24 of hundreds of radians), so its remainder is carried along and applied as a small rotation.
__device__ __forceinline__ void rot_angle(int pos, float2 f, float* sn, float* cs) {
  const float a = (float)pos * f.x;
  const float r = fmaf((float)pos, f.x, -a) + (float)pos * f.y;
  float s, c;
  sincosf(a, &s, &c);
  *sn = fmaf(r, c, s);
  *cs = fmaf(-r, s, c);
}

// one element of a normed and rotated query or key head: src points at the head's raw values, w at
// its norm weights, rinv is 1 / rms of the whole projection, cs holds (cos, sin) of the position
__device__ __forceinline__ float rot_elem(const AttnP& p, const float* src, const float* w, float rinv, const float2* cs,
                                          int d) {
  if (d >= 2 * p.pairs) return src[d] * rinv * w[d];
  const int e = d & ~1;
  const float u = src[e] * rinv * w[e], v = src[e + 1] * rinv * w[e + 1];
  const float2 t = cs[d >> 1];
  return (d & 1) ? v * t.x + u * t.y : u * t.x - v * t.y;
}
constexpr int MX_PAIRS = 512;   // most rotated pairs of a head
__device__ __forceinline__ void rot_table(const AttnP& p, int pos, float2* cs) {
  for (int i = threadIdx.x; i < p.pairs; i += blockDim.x) rot_angle(pos, p.inv_freq[i], &cs[i].y, &cs[i].x);
}

constexpr int MX_THREADS = 256;
constexpr int MX_TK = 256;      // keys per tile

// Attention of up to RM query heads of one key/value head over the visible indices [t0, t1) of one
// position: qs [RM][Dp] in shared memory, scores through sc [RM][MX_TK], result (unnormalised) in
// os [RM][Ep], running maxima and sums in ml [2][RM].  The whole block; barriers inside.
template <typename KT, int RM>
__device__ void attn_range(const AttnP& p, const float* qs, int g, const Visible& vis, int t0, int t1, float* sc,
                           float* os, float* ml) {
  constexpr int CE = Vec16<KT>::N;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const KT* K = (const KT*)p.K + (size_t)g * p.cap * p.Dp;
  const KT* V = (const KT*)p.V + (size_t)g * p.cap * p.Vs;
  float* corr = ml + 2 * RM;
  if (tid < RM) { ml[tid] = -3.0e38f; ml[RM + tid] = 0.f; }
  const int nc2 = p.Ep / 2, ngrp = MX_THREADS / nc2 < 1 ? 1 : MX_THREADS / nc2;
  const int grp = tid / nc2, col = (tid - grp * nc2) * 2;
  const bool pv = grp < ngrp;
  float acc[RM][2];
#pragma unroll
  for (int r = 0; r < RM; r++) acc[r][0] = acc[r][1] = 0.f;
  for (int tb = t0; tb < t1; tb += MX_TK) {
    const int n = t1 - tb < MX_TK ? t1 - tb : MX_TK;
    __syncthreads();
    for (int kb = 0; kb < n; kb += MX_THREADS / 8) {
      const int kk = kb + (tid >> 3);
      float s[RM];
#pragma unroll
      for (int r = 0; r < RM; r++) s[r] = 0.f;
      if (kk < n) {
        const KT* row = K + (size_t)kv_slot(p, visible_pos(vis, tb + kk)) * p.Dp;
        for (int c = lane & 7; c < p.Dp / CE; c += 8) {
          float f[CE];
          widen16(*(const uint4*)(row + c * CE), f, (const KT*)nullptr);
#pragma unroll
          for (int r = 0; r < RM; r++)
#pragma unroll
            for (int e = 0; e < CE; e += 4) {
              const float4 q4 = *(const float4*)(qs + r * p.Dp + c * CE + e);
              s[r] = fmaf(f[e], q4.x, s[r]); s[r] = fmaf(f[e + 1], q4.y, s[r]);
              s[r] = fmaf(f[e + 2], q4.z, s[r]); s[r] = fmaf(f[e + 3], q4.w, s[r]);
            }
        }
      }
#pragma unroll
      for (int r = 0; r < RM; r++) {
        s[r] += __shfl_xor_sync(0xffffffffu, s[r], 1);
        s[r] += __shfl_xor_sync(0xffffffffu, s[r], 2);
        s[r] += __shfl_xor_sync(0xffffffffu, s[r], 4);
        if (kk < n && (lane & 7) == (r & 7)) sc[r * MX_TK + kk] = s[r] * p.scale;
      }
    }
    __syncthreads();
    for (int r = warp; r < RM; r += MX_THREADS / 32) {
      float m = ml[r];
      const float old = m;
      for (int k = lane; k < n; k += 32) m = fmaxf(m, sc[r * MX_TK + k]);
      m = warp_max(m);
      float l = 0.f;
      for (int k = lane; k < n; k += 32) {
        const float e = expf(sc[r * MX_TK + k] - m);
        sc[r * MX_TK + k] = e;
        l += e;
      }
      l = warp_sum(l);
      if (lane == 0) {
        const float cr = expf(old - m);
        corr[r] = cr; ml[r] = m; ml[RM + r] = ml[RM + r] * cr + l;
      }
    }
    __syncthreads();
    if (pv) {
#pragma unroll
      for (int r = 0; r < RM; r++) { acc[r][0] *= corr[r]; acc[r][1] *= corr[r]; }
#pragma unroll 4
      for (int k = grp; k < n; k += ngrp) {
        float a, b;
        load2(V + (size_t)kv_slot(p, visible_pos(vis, tb + k)) * p.Vs + col, a, b);
#pragma unroll
        for (int r = 0; r < RM; r++) {
          const float w = sc[r * MX_TK + k];
          acc[r][0] = fmaf(w, a, acc[r][0]);
          acc[r][1] = fmaf(w, b, acc[r][1]);
        }
      }
    }
  }
  for (int q = 0; q < ngrp; q++) {
    __syncthreads();
    if (pv && grp == q) {
#pragma unroll
      for (int r = 0; r < RM; r++) {
        float* o = os + r * p.Ep + col;
        o[0] = q ? o[0] + acc[r][0] : acc[r][0];
        o[1] = q ? o[1] + acc[r][1] : acc[r][1];
      }
    }
  }
  __syncthreads();
}

// convolution input of channel c at `pos`, silu behind it.  cur points at channel 0 of the row of
// `pos` in the projected rows (row stride ld), of which `have` earlier rows belong to this pass.
__device__ __forceinline__ float conv_silu(const ConvP& p, const float* cur, long long ld, int have, int pos, int c) {
  float y = p.b ? p.b[c] : 0.f;
  for (int a = 0; a < p.taps; a++) {
    const int d = p.taps - 1 - a, q = pos - d;
    if (q < 0) continue;
    const float x = d <= have ? cur[c - (long long)d * ld] : p.ring[(size_t)(q % p.taps) * p.C + c];
    y = fmaf(p.w[(size_t)c * p.taps + a], x, y);
  }
  return silu_f(y);
}

// exp(-x) of a decay that is applied once per token: near 1 it is rounded from an exact complement,
// so that hundreds of factors do not add up the exponential's own last-place error.
__device__ __forceinline__ float decay_of(float x) { return x < 0.5f ? 1.0f + expm1f(-x) : expf(-x); }

// step size and decay rate of head h: (beta, -log g) of the delta rule, (dt, -log decay) of ssd
__device__ __forceinline__ float2 recur_gates(const RecurP& p, const float* row, int h) {
  if (p.kind == MIX_DELTA)
    return make_float2(sigmoid_f(row[p.ob + h]),
                       expf(p.A_log[h]) * softplus_f(row[p.oa_ + h] + p.dt_bias[h]));
  const float dt = softplus_f(row[p.ob + h] + p.dt_bias[h]);
  return make_float2(dt, expf(p.A_log[h]) * dt);
}

// -log of a gla decay: z is the sum behind the decay's projections
__device__ __forceinline__ float gla_rate(float z, float tau) { return softplus_f(-z) / tau; }

#endif  // __CUDACC__

// launchers (mixers.cu, rows.cu)
int mixers_decode_launch(const AttnP* attn, const RecurP* rec, int n_rec, const float* proj, float* out,
                         const unsigned* d_pos, bool kv_bf16, cudaStream_t s);
int attn_rows_prep_launch(const AttnP& p, const float* proj, long long ld, int rows, int pos0, void* q, bool bf16,
                          cudaStream_t s);
int attn_rows_launch(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda, int rows,
                     int pos0, bool bf16, cudaStream_t s);
// the same on the tensor pipe (attn_window.cu): bf16, widths up to 128
bool attn_window_eligible(const AttnP& p);
// the kernel behind it: where the rows of queries, keys (a part of their own and a shared part behind it)
// and values lie; strides in elements, widths multiples of 8
struct AttnTiles {
  const void *q, *k, *k2, *v;
  long long q_row, q_head, k_row, k_head, k2_row, v_row, v_head;
  int kw, k2w, vw;             // widths of the key parts and of a value row; a query has kw + k2w
  int H, R, E;                 // heads, heads on one key head, value width
  int window, keep, ring;
  float scale, out_scale;
  const float* gate;           // [row][gate_row], head h at h * E; NULL: none
  long long gate_row;
};
bool attn_tiles_eligible(int qk_width, int v_width);
int attn_tiles_launch(const AttnTiles& t, void* out, long long ldo, int rows, int pos0, cudaStream_t s);
int attn_window_launch(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda,
                       int rows, int pos0, cudaStream_t s);
// Convolutions, step sizes and rates of a pass, in one of two forms: f32 with the delta rule's unit
// queries and keys (norms NULL), for the token-by-token scan; or bf16 as the convolutions leave them,
// with the factors that make queries and keys unit vectors apart ([rows][G] query, key), for the chunks.
int recur_rows_conv_launch(const RecurP& p, const float* proj, long long ld, int rows, int pos0, void* conv,
                           float2* gates, float2* norms, bool chunked, cudaStream_t s);
// gla: conv is the projected rows (stride ld), gates the rates [rows][H * D]
int recur_rows_scan_launch(const RecurP& p, const float* conv, long long ld, const void* gates, float* o, int rows,
                           int pos0, cudaStream_t s);
int recur_rows_finish_launch(const RecurP& p, const float* o, const void* conv, bool conv_bf16, const float* proj,
                             long long ld, void* act, long long lda, int norm_groups, int rows, bool bf16, cudaStream_t s);
// the recurrence in chunks on the tensor pipe (recur_chunk.cu)
bool recur_chunk_eligible(const RecurP& p);
size_t recur_chunk_scratch_bytes(const RecurP& p, int rows);
int recur_chunk_launch(const RecurP& p, const void* conv, const float2* gates, const float2* norms, void* scratch,
                       float* o, int rows, int pos0, cudaStream_t s);
// gated linear attention of a pass (recur_gla.cu): rates of every row and key channel, then the recurrence
// token by token or in chunks on the tensor pipe (bf16)
int gla_rates_launch(const RecurP& p, const float* proj, long long ld, float* rates, int rows, cudaStream_t s);
bool gla_chunk_eligible(const RecurP& p);
size_t gla_chunk_scratch_bytes(const RecurP& p, int rows);
int gla_chunk_launch(const RecurP& p, const float* proj, long long ld, const float* rates, void* scratch, float* o,
                     int rows, int pos0, cudaStream_t s);

// latent attention (attn_latent.cu).  `rows` positions from *d_pos (one token) or from pos0:
//   prep     (prompt pass) normed query latents, kept rows
//   absorb   queries against the latent, rotated; with d_pos the token's kept row
//   attend   weighted latents of key ranges, with their maxima and sums
//   fold     ranges merged, values, gate
// or, for many rows in bf16: q_rows (rotated queries) and attn_tiles on expanded keys and values
size_t latent_part_floats(const LatentP& p, int rows, int splits);
int latent_splits(const LatentP& p, int rows);
int latent_prep_launch(const LatentP& p, const float* proj, long long ld, int rows, int pos0, void* qlat, bool bf16,
                       cudaStream_t s);
int latent_absorb_launch(const LatentP& p, const float* q, long long ldq, const float* proj, void* qa, int rows,
                         const unsigned* d_pos, int pos0, bool bf16, cudaStream_t s);
int latent_attend_launch(const LatentP& p, const void* qa, float* part, int rows, int splits, const unsigned* d_pos,
                         int pos0, bool bf16, cudaStream_t s);
int latent_fold_launch(const LatentP& p, const float* part, int splits, const float* proj, long long ld, void* act,
                       long long lda, int rows, const unsigned* d_pos, int pos0, bool bf16, bool act_bf16, cudaStream_t s);
int latent_q_rows_launch(const LatentP& p, const float* q, long long ldq, void* out, int rows, int pos0, cudaStream_t s);

int rms_rows_launch(const float* x, long long ldx, const float* w, void* out, long long ldo, int n, float eps,
                    float scale, int rows, bool bf16, cudaStream_t s);
// x += norm(y) (y NULL: x as it is), and the result as the next product's operand
int residual_rows_launch(float* x, const float* y, const float* w, void* out, long long ldo, int n, float eps, int rows,
                         bool bf16, cudaStream_t s);
int embed_scaled_launch(const void* embed, const int* ids, float* x, int width, long long ld, float scale, int rows,
                        bool bf16, cudaStream_t s);
int gather_rows_launch(const float* x, const int* idx, float* out, int width, int rows, cudaStream_t s);
int glu_rows_launch(const float* gu, float* out, int ff, float limit, int rows, cudaStream_t s);
int relu2_rows_launch(const float* u, float* out, int ff, int rows, cudaStream_t s);

// one-row matrix product with its neighbours fused (gemv_rows.cu)
struct RowGemv {
  const float* x;            // [K]
  const void* W;             // [N][ldw]
  int N, K;
  long long ldw;
  // RMS norm of x[n_off, n_off + n_len) in n_groups equal parts, times nw and nscale, in front of
  // the product (nw NULL: none)
  const float* nw;
  int n_off, n_len, n_groups;
  float eps, nscale;
  const float* gate;         // [n_len] the normed part times silu(gate) (NULL: none)
  // a residual in front of it all: the row becomes res + norm(x) * rn, block 0 leaves it in xout
  const float *res, *rn;
  float* xout;
  float* y;
  int epi;                   // 0 y = , 1 y += , 2 y[j] = glu(row 2j, row 2j + 1), 3 y = relu2
  float limit;
};
int row_gemv_launch(DeviceCtx* c, const RowGemv& p, bool bf16, cudaStream_t s);

bool gemm_bf16_tc_eligible(const void* a, long long lda, const void* w, long long ldw);
int gemm_bf16_tc_launch(DeviceCtx* c, const void* a, long long lda, const void* w, long long ldw, float* C,
                        long long ldc, void* O, long long ldo, int M, int N, int K, int epi, float limit,
                        cudaStream_t s);

}  // namespace tlb
