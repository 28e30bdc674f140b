// Prompt attention of the layer-stack decoder on the tensor pipe: sliding window with the first tokens
// kept, grouped heads, bf16 queries / keys / values, f32 scores, weights and accumulation, with the
// sigmoid output gate in the epilogue.
//
// One CTA = 64 query rows of one head (4 warps of 16 rows) walking the keys its rows can see: the kept
// positions first, then the window of its first row up to its last row, 64 keys a tile, fetched row by
// row from the cache's kept slots and ring with 16-byte cp.async into a double buffer.  Scores and
// products are mma.sync m16n8k16 with bf16 operands; a tile that every row of a warp sees whole skips
// the mask.  Widths up to 128 (rounded up to 32 / 64 / 96 / 128 with zero columns).
#include "mixers.cuh"

namespace tlb {

namespace {

constexpr int AW_M = 64, AW_N = 64, AW_THREADS = 128;

__device__ __forceinline__ void aw_cp16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void aw_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void aw_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void aw_ldm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void aw_ldm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void aw_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t aw_pack(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *(const uint32_t*)&h;
}

template <int DM>
struct AwSmem {
  static constexpr int LD = DM + 8;                       // row stride in elements
  static constexpr size_t Q = 0;
  static constexpr size_t K = Q + (size_t)AW_M * LD * 2;
  static constexpr size_t V = K + (size_t)2 * AW_N * LD * 2;
  static constexpr size_t TOTAL = V + (size_t)2 * AW_N * LD * 2;
};

template <int DM>
__global__ void __launch_bounds__(AW_THREADS, 2)
    attn_window_kernel(const __grid_constant__ AttnP p, const __nv_bfloat16* __restrict__ q,
                       const float* __restrict__ proj, long long ld, __nv_bfloat16* __restrict__ act, long long lda,
                       int rows, int pos0) {
  using S = AwSmem<DM>;
  constexpr int LD = S::LD, CH = DM / 8;
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* qs = (__nv_bfloat16*)(smem + S::Q);
  __nv_bfloat16* ks = (__nv_bfloat16*)(smem + S::K);
  __nv_bfloat16* vs = (__nv_bfloat16*)(smem + S::V);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = (gridDim.x - 1 - blockIdx.x) * AW_M, h = blockIdx.y, g = h / (p.H / p.G);
  const int nrow = rows - r0 < AW_M ? rows - r0 : AW_M;
  const int dch = p.Dp / 8, ech = p.Ep / 8;
  // zero columns behind the widths: never written again
  for (int i = tid; i < (AW_M + 4 * AW_N) * (LD / 8); i += AW_THREADS) ((uint4*)smem)[i] = make_uint4(0, 0, 0, 0);
  pdl_wait();
  pdl_launch_dependents();
  __syncthreads();
  for (int i = tid; i < nrow * dch; i += AW_THREADS) {
    const int r = i / dch, c = i - r * dch;
    aw_cp16(qs + r * LD + c * 8, q + ((size_t)(r0 + r) * p.H + h) * p.Dp + c * 8, true);
  }
  // what the block's rows can see: kept positions in front of the first row's window, then the window
  const int pf = pos0 + r0, pl = pf + nrow - 1;
  Visible vis;
  vis.lo = pf + 1 > p.window ? pf + 1 - p.window : 0;
  vis.kept = p.keep < vis.lo ? p.keep : vis.lo;
  vis.n = vis.kept + pl + 1 - vis.lo;
  const __nv_bfloat16* K = (const __nv_bfloat16*)p.K + (size_t)g * p.cap * p.Dp;
  const __nv_bfloat16* V = (const __nv_bfloat16*)p.V + (size_t)g * p.cap * p.Ep;
  auto fetch = [&](int tile, int buf) {
    // two threads a key row, one half of its chunks each
    const int r = tid >> 1, half = tid & 1, t = tile * AW_N + r;
    const bool on = t < vis.n;
    const size_t slot = kv_slot(p, on ? visible_pos(vis, t) : 0);
    const __nv_bfloat16 *kr = K + slot * p.Dp, *vr = V + slot * p.Ep;
    __nv_bfloat16 *kd = ks + (buf * AW_N + r) * LD, *vd = vs + (buf * AW_N + r) * LD;
#pragma unroll
    for (int i = 0; i < CH / 2; i++) {
      const int c = 2 * i + half;
      if (c < dch) aw_cp16(kd + c * 8, kr + c * 8, on);
      if (c < ech) aw_cp16(vd + c * 8, vr + c * 8, on);
    }
  };
  const int ntile = (vis.n + AW_N - 1) / AW_N;
  fetch(0, 0);
  aw_commit();
  float o[DM / 8][4];
#pragma unroll
  for (int i = 0; i < DM / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-1.0e30f, -1.0e30f}, l[2] = {0.f, 0.f};
  uint32_t qf[DM / 16][4];
  const int wr = warp * 16, row_a = wr + (lane >> 2), col_a = (lane & 3) * 2;
  const int pa = pf + row_a, pb = pa + 8;                 // positions of the thread's two rows
  const int wp0 = pf + wr, wp1 = wp0 + 15;                // of the warp's
  const float sl2 = p.scale * 1.4426950408889634f;
  for (int t = 0; t < ntile; t++) {
    const int buf = t & 1;
    if (t + 1 < ntile) {
      fetch(t + 1, buf ^ 1);
      aw_commit();
      aw_wait<1>();
    } else {
      aw_wait<0>();
    }
    __syncthreads();
    if (t == 0) {
#pragma unroll
      for (int k = 0; k < DM / 16; k++)
        aw_ldm4(qf[k], qs + (wr + (lane & 15)) * LD + k * 16 + (lane >> 4) * 8);
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
      const __nv_bfloat16* kb = ks + buf * AW_N * LD;
#pragma unroll
      for (int k = 0; k < DM / 16; k++)
#pragma unroll
        for (int n = 0; n < 4; n++) {
          uint32_t b[4];
          aw_ldm4(b, kb + (n * 16 + (lane & 7) + ((lane >> 4) << 3)) * LD + k * 16 + ((lane >> 3) & 1) * 8);
          aw_mma(s[2 * n], qf[k], b[0], b[1]);
          aw_mma(s[2 * n + 1], qf[k], b[2], b[3]);
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
        for (int i = 0; i < DM / 8; i++) { o[i][2 * e] *= c; o[i][2 * e + 1] *= c; }
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
      const __nv_bfloat16* vb = vs + buf * AW_N * LD;
#pragma unroll
      for (int k = 0; k < 4; k++)
#pragma unroll
        for (int n = 0; n < DM / 16; n++) {
          uint32_t b[4];
          aw_ldm4t(b, vb + (k * 16 + (lane & 15)) * LD + n * 16 + (lane >> 4) * 8);
          aw_mma(o[2 * n], pf_[k], b[0], b[1]);
          aw_mma(o[2 * n + 1], pf_[k], b[2], b[3]);
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
    const float* gate = proj + (size_t)(r0 + r) * ld + p.og + h * p.E;
    __nv_bfloat16* dst = act + (size_t)(r0 + r) * lda + p.oa + h * p.E;
#pragma unroll
    for (int n = 0; n < DM / 8; n++) {
      const int c = n * 8 + col_a;
      const float a = o[n][2 * e] * inv, b = o[n][2 * e + 1] * inv;
      if ((p.E & 1) == 0) {
        if (c < p.E) {
          const float2 gt = *(const float2*)(gate + c);
          *(uint32_t*)(dst + c) = aw_pack(a * sigmoid_f(gt.x), b * sigmoid_f(gt.y));
        }
      } else {
        if (c < p.E) dst[c] = __float2bfloat16_rn(a * sigmoid_f(gate[c]));
        if (c + 1 < p.E) dst[c + 1] = __float2bfloat16_rn(b * sigmoid_f(gate[c + 1]));
      }
    }
  }
}

template <int DM>
int aw_launch(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda, int rows,
              int pos0, cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(attn_window_kernel<DM>, (int)AwSmem<DM>::TOTAL, done);
  if (rc) return rc;
  LaunchCfg lc(dim3((rows + AW_M - 1) / AW_M, p.H), dim3(AW_THREADS), AwSmem<DM>::TOTAL, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, attn_window_kernel<DM>, p, (const __nv_bfloat16*)q, proj, ld,
                              (__nv_bfloat16*)act, lda, rows, pos0));
  return TLB_OK;
}

}  // namespace

bool attn_window_eligible(const AttnP& p) { return p.Dp <= 128 && p.Ep <= 128; }

int attn_window_launch(const AttnP& p, const void* q, const float* proj, long long ld, void* act, long long lda,
                       int rows, int pos0, cudaStream_t s) {
  const int w = p.Dp > p.Ep ? p.Dp : p.Ep;
  if (w <= 32) return aw_launch<32>(p, q, proj, ld, act, lda, rows, pos0, s);
  if (w <= 64) return aw_launch<64>(p, q, proj, ld, act, lda, rows, pos0, s);
  if (w <= 96) return aw_launch<96>(p, q, proj, ld, act, lda, rows, pos0, s);
  return aw_launch<128>(p, q, proj, ld, act, lda, rows, pos0, s);
}

}  // namespace tlb
