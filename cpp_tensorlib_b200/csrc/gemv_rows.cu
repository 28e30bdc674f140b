// One-row matrix product of the layer-stack decoder, y = W . f(x), with its neighbours fused: an
// RMS norm (whole row, or a segment in equal parts) on the staged activation in front, a residual
// add or the clipped gated unit behind.  W is bf16 or f32 row-major, everything else f32.
//
// HBM bound.  A warp owns one row, or two adjacent rows (gate and up interleaved), and keeps eight
// 16-byte loads in flight plus the next eight; the first eight are issued BEFORE the wait for the
// preceding kernel, so a launch's weight stream starts under its predecessor's tail.
#include "mixers.cuh"

namespace tlb {

namespace {

constexpr int RG_WARPS = 8;

__device__ __forceinline__ uint4 rg_ld(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

template <typename WT, int R>
__global__ void __launch_bounds__(RG_WARPS * 32, 2) row_gemv_kernel(const __grid_constant__ RowGemv p) {
  constexpr int CE = Vec16<WT>::N, U = 8 / R;
  extern __shared__ __align__(16) float xs[];   // [ldw], zero behind K
  __shared__ float red[33];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int chunks = (int)(p.ldw / CE), groups = (p.N + R - 1) / R, stride = gridDim.x * RG_WARPS;
  const WT* W = (const WT*)p.W;
  int rg = blockIdx.x * RG_WARPS + warp, cb = 0;
  uint4 cur[R][U], nxt[R][U];
  auto fetch = [&](uint4 (&w)[R][U], int g, int b) {
#pragma unroll
    for (int r = 0; r < R; r++) {
      const WT* row = W + (size_t)(g * R + r < p.N ? g * R + r : p.N - 1) * p.ldw;
#pragma unroll
      for (int u = 0; u < U; u++) {
        const int c = b + lane + 32 * u;
        w[r][u] = c < chunks ? rg_ld(row + (size_t)c * CE) : make_uint4(0, 0, 0, 0);
      }
    }
  };
  if (rg < groups) fetch(cur, rg, 0);
  pdl_wait();
  pdl_launch_dependents();
  for (int i = tid; i < p.ldw; i += RG_WARPS * 32) xs[i] = i < p.K ? p.x[i] : 0.f;
  if (p.nw) {
    const int m = p.n_len / p.n_groups;
    for (int g = 0; g < p.n_groups; g++) {
      float* seg = xs + p.n_off + g * m;
      float sq = 0.f;
      __syncthreads();
      for (int i = tid; i < m; i += RG_WARPS * 32) sq = fmaf(seg[i], seg[i], sq);
      sq = block_sum(sq, red);
      const float s = rsqrtf(sq / m + p.eps) * p.nscale;
      for (int i = tid; i < m; i += RG_WARPS * 32) seg[i] = seg[i] * s * p.nw[g * m + i];
    }
  }
  __syncthreads();
  float acc[R][2];
#pragma unroll
  for (int r = 0; r < R; r++) acc[r][0] = acc[r][1] = 0.f;
  while (rg < groups) {
    int ng = rg, nb = cb + 32 * U;
    if (nb >= chunks) { ng += stride; nb = 0; }
    if (ng < groups) fetch(nxt, ng, nb);
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int c = cb + lane + 32 * u;
      if (c < chunks) {
        float x[CE];
#pragma unroll
        for (int e = 0; e < CE; e += 4) {
          const float4 v = *(const float4*)(xs + (size_t)c * CE + e);
          x[e] = v.x; x[e + 1] = v.y; x[e + 2] = v.z; x[e + 3] = v.w;
        }
#pragma unroll
        for (int r = 0; r < R; r++) {
          float w[CE];
          widen16(cur[r][u], w, (const WT*)nullptr);
#pragma unroll
          for (int e = 0; e < CE; e++) acc[r][e & 1] = fmaf(w[e], x[e], acc[r][e & 1]);
        }
      }
    }
    if (ng != rg) {
      float a[R];
#pragma unroll
      for (int r = 0; r < R; r++) {
        a[r] = warp_sum(acc[r][0] + acc[r][1]);
        acc[r][0] = acc[r][1] = 0.f;
      }
      if (lane == 0) {
        if (p.epi == 2) {
          if (R == 2) p.y[rg] = glu_clipped(a[0], a[R - 1], p.limit);
        } else {
#pragma unroll
          for (int r = 0; r < R; r++) {
            const int n = rg * R + r;
            if (n < p.N) p.y[n] = p.epi == 1 ? p.y[n] + a[r] : a[r];
          }
        }
      }
    }
    rg = ng;
    cb = nb;
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
      for (int u = 0; u < U; u++) cur[r][u] = nxt[r][u];
  }
}

template <typename WT, int R>
int rg_launch(DeviceCtx* c, const RowGemv& p, cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(row_gemv_kernel<WT, R>, 220 * 1024, done);
  if (rc) return rc;
  const int need = ((p.N + R - 1) / R + RG_WARPS - 1) / RG_WARPS;
  const int ctas = need < 2 * c->sm_count ? need : 2 * c->sm_count;
  LaunchCfg lc(dim3(ctas), dim3(RG_WARPS * 32), (size_t)p.ldw * sizeof(float), s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, row_gemv_kernel<WT, R>, p));
  return TLB_OK;
}

// ---- row ops of the prompt pass --------------------------------------------------------------
template <typename OT>
__global__ void __launch_bounds__(256) rms_rows_kernel(const float* __restrict__ x, long long ldx,
                                                       const float* __restrict__ w, OT* __restrict__ out, long long ldo,
                                                       int n, float eps) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const float* row = x + (size_t)blockIdx.x * ldx;
  OT* dst = out + (size_t)blockIdx.x * ldo;
  float sq = 0.f;
  for (int i = threadIdx.x; i < n; i += 256) sq = fmaf(row[i], row[i], sq);
  sq = block_sum(sq, red);
  const float r = rsqrtf(sq / n + eps);
  for (int i = threadIdx.x; i < n; i += 256) put(dst + i, row[i] * r * w[i]);
}

template <typename WT>
__global__ void embed_scaled_kernel(const WT* __restrict__ embed, long long ld, const int* __restrict__ ids,
                                    float* __restrict__ x, int width, float scale) {
  pdl_wait();
  pdl_launch_dependents();
  const WT* src = embed + (size_t)ids[blockIdx.x] * ld;
  for (int i = threadIdx.x; i < width; i += blockDim.x) x[(size_t)blockIdx.x * width + i] = to_f(src[i]) * scale;
}

__global__ void gather_rows_kernel(const float* __restrict__ x, const int* __restrict__ idx, float* __restrict__ out,
                                   int width) {
  pdl_wait();
  pdl_launch_dependents();
  const float* src = x + (size_t)idx[blockIdx.x] * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) out[(size_t)blockIdx.x * width + i] = src[i];
}

__global__ void glu_rows_kernel(const float* __restrict__ gu, float* __restrict__ out, long long n, float limit) {
  pdl_wait();
  pdl_launch_dependents();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const float2 v = ((const float2*)gu)[i];
    out[i] = glu_clipped(v.x, v.y, limit);
  }
}

}  // namespace

int row_gemv_launch(DeviceCtx* c, const RowGemv& p, bool bf16, cudaStream_t s) {
  if (p.ldw * (long long)sizeof(float) > 216 * 1024)
    return set_error(TLB_ERR_UNSUPPORTED, "row_gemv: the activation row does not fit the shared-memory stage");
  // two rows a warp where the rows come in pairs, or where there are enough of them to fill the SMs
  const bool two = p.epi == 2 || p.N >= 2 * 2 * c->sm_count * RG_WARPS;
  if (bf16) return two ? rg_launch<__nv_bfloat16, 2>(c, p, s) : rg_launch<__nv_bfloat16, 1>(c, p, s);
  return two ? rg_launch<float, 2>(c, p, s) : rg_launch<float, 1>(c, p, s);
}

int rms_rows_launch(const float* x, long long ldx, const float* w, void* out, long long ldo, int n, float eps, int rows,
                    bool bf16, cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
  if (bf16) TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, rms_rows_kernel<__nv_bfloat16>, x, ldx, w, (__nv_bfloat16*)out, ldo, n, eps));
  else TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, rms_rows_kernel<float>, x, ldx, w, (float*)out, ldo, n, eps));
  return TLB_OK;
}

int embed_scaled_launch(const void* embed, const int* ids, float* x, int width, long long ld, float scale, int rows,
                        bool bf16, cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
  if (bf16) TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, embed_scaled_kernel<__nv_bfloat16>, (const __nv_bfloat16*)embed, ld, ids, x, width, scale));
  else TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, embed_scaled_kernel<float>, (const float*)embed, ld, ids, x, width, scale));
  return TLB_OK;
}

int gather_rows_launch(const float* x, const int* idx, float* out, int width, int rows, cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, gather_rows_kernel, x, idx, out, width));
  return TLB_OK;
}

int glu_rows_launch(const float* gu, float* out, int ff, float limit, int rows, cudaStream_t s) {
  const long long n = (long long)rows * ff;
  const long long b = (n + 255) / 256;
  LaunchCfg lc(dim3((unsigned)(b < 148 * 16 ? b : 148 * 16)), dim3(256), 0, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, glu_rows_kernel, gu, out, n, limit));
  return TLB_OK;
}

}  // namespace tlb
