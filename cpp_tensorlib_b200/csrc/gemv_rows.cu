// One-row matrix product of the layer-stack decoder, y = W . f(x), with its neighbours fused: on the
// staged activation in front, the residual sum that a norm of the preceding sublayer's output ends in,
// an RMS norm (whole row, or a segment in equal parts) and a silu gate; a residual add, the clipped
// gated unit or the square of relu behind.  W is bf16 or f32 row-major, everything else f32.
//
// HBM bound.  A stream of ks adjacent warps owns one row, or two adjacent rows (gate and up
// interleaved), each warp its own part of K; ks is picked on the host so that the streams of all SMs
// come out even.  Every warp keeps eight 16-byte loads in flight plus the next eight; the first eight
// are issued BEFORE the wait for the preceding kernel, so a launch's weight stream starts under its
// predecessor's tail.  Weights are marked evict-first in the L2: a token streams gigabytes of them
// once, and what every launch needs again -- instructions, states, activations -- should stay.
#include "mixers.cuh"

namespace tlb {

namespace {

constexpr int RG_WARPS = 8;

__device__ __forceinline__ uint4 rg_ld(const void* p, uint64_t pol) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.L2::cache_hint.v4.u32 {%0,%1,%2,%3}, [%4], %5;"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p), "l"(pol));
  return v;
}

// x into xs [ldw], zero behind K; returns this thread's share of its sum of squares.  Kept short: a
// launch runs this code once, from a cold instruction cache.
__device__ __forceinline__ float rg_stage(const RowGemv& p, float* xs) {
  float sq = 0.f;
  const int k4 = ((uintptr_t)p.x & 15) ? 0 : p.K / 4;   // rows of an odd width go one by one
  for (int i0 = threadIdx.x; i0 < k4; i0 += 4 * RG_WARPS * 32) {
    float4 v[4];
#pragma unroll
    for (int u = 0; u < 4; u++)
      if (i0 + u * RG_WARPS * 32 < k4) v[u] = ((const float4*)p.x)[i0 + u * RG_WARPS * 32];
#pragma unroll
    for (int u = 0; u < 4; u++)
      if (i0 + u * RG_WARPS * 32 < k4) {
        ((float4*)xs)[i0 + u * RG_WARPS * 32] = v[u];
        sq = fmaf(v[u].x, v[u].x, fmaf(v[u].y, v[u].y, fmaf(v[u].z, v[u].z, fmaf(v[u].w, v[u].w, sq))));
      }
  }
#pragma unroll 1
  for (int i = 4 * k4 + threadIdx.x; i < p.ldw; i += RG_WARPS * 32) {
    const float x = i < p.K ? p.x[i] : 0.f;
    xs[i] = x;
    sq = fmaf(x, x, sq);
  }
  return sq;
}

// the preceding sublayer's output, normed, added to the residual: every block computes the row, block 0
// leaves it for the launches behind.  Returns the thread's share of the new row's sum of squares.
__device__ __forceinline__ float rg_residual(const RowGemv& p, float* xs, float sq, float* red) {
  const float s = rsqrtf(block_sum(sq, red) / p.K + p.eps);
  sq = 0.f;
#pragma unroll 8
  for (int i = threadIdx.x; i < p.K; i += RG_WARPS * 32) {
    const float v = fmaf(xs[i] * s, p.rn[i], p.res[i]);
    xs[i] = v;
    if (p.xout && blockIdx.x == 0) p.xout[i] = v;
    sq = fmaf(v, v, sq);
  }
  return sq;
}

// the norm in place: the whole row by the block, a segment in parts a warp each
__device__ __forceinline__ void rg_norm(const RowGemv& p, float* xs, float sq, float* red) {
  const int tid = threadIdx.x, lane = tid & 31;
  if (p.n_groups == 1 && p.n_len == p.K) {
    const float s = rsqrtf(block_sum(sq, red) / p.K + p.eps) * p.nscale;
#pragma unroll 4
    for (int i = tid; i < p.K; i += RG_WARPS * 32) xs[i] *= p.gate ? s * p.nw[i] * silu_f(p.gate[i]) : s * p.nw[i];
    return;
  }
  __syncthreads();
  const int m = p.n_len / p.n_groups;
#pragma unroll 1
  for (int g = tid >> 5; g < p.n_groups; g += RG_WARPS) {
    float* seg = xs + p.n_off + g * m;
    float q = 0.f;
#pragma unroll 4
    for (int i = lane; i < m; i += 32) q = fmaf(seg[i], seg[i], q);
    const float s = rsqrtf(warp_sum(q) / m + p.eps) * p.nscale;
#pragma unroll 4
    for (int i = lane; i < m; i += 32)
      seg[i] *= p.gate ? s * p.nw[g * m + i] * silu_f(p.gate[g * m + i]) : s * p.nw[g * m + i];
  }
}

template <int R>
__device__ __forceinline__ void rg_emit(const RowGemv& p, int rg, const float (&a)[R]) {
  if (p.epi == 2) {
    if (R == 2) p.y[rg] = glu_clipped(a[0], a[R - 1], p.limit);
    return;
  }
#pragma unroll
  for (int r = 0; r < R; r++) {
    const int n = rg * R + r;
    if (n < p.N) p.y[n] = p.epi == 1 ? p.y[n] + a[r] : (p.epi == 3 ? relu2(a[r]) : a[r]);
  }
}

template <typename WT, int R>
__global__ void __launch_bounds__(RG_WARPS * 32, 2) row_gemv_kernel(const __grid_constant__ RowGemv p, int ks) {
  constexpr int CE = Vec16<WT>::N, U = 8 / R;
  extern __shared__ __align__(16) float xs[];   // [ldw], then the streams' partial sums
  __shared__ float red[33];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int groups = (p.N + R - 1) / R, ns = RG_WARPS / ks, stream = warp / ks, sub = warp - stream * ks;
  const int stride = gridDim.x * ns, chunks = (int)(p.ldw / CE), per = (chunks + ks - 1) / ks;
  const int c_lo = sub * per, c_hi = c_lo + per < chunks ? c_lo + per : chunks;
  float* part = xs + p.ldw;                     // [local group][stream][R][ks]
  const WT* W = (const WT*)p.W;
  const uint64_t pol = l2_evict_first_policy();
  int rg = blockIdx.x * ns + stream, cb = c_lo, loc = 0;
  uint4 cur[R][U], nxt[R][U];
  auto fetch = [&](uint4 (&w)[R][U], int g, int b) {
#pragma unroll
    for (int r = 0; r < R; r++) {
      const WT* row = W + (size_t)(g * R + r < p.N ? g * R + r : p.N - 1) * p.ldw;
#pragma unroll
      for (int u = 0; u < U; u++) {
        const int c = b + lane + 32 * u;
        w[r][u] = c < c_hi ? rg_ld(row + (size_t)c * CE, pol) : make_uint4(0, 0, 0, 0);
      }
    }
  };
  if (rg < groups) fetch(cur, rg, cb);
  if (p.nw)   // the norm's weights into the L2
    for (int i = tid * 32; i < p.n_len; i += RG_WARPS * 32 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.nw + i));
  if (p.rn)
    for (int i = tid * 32; i < p.K; i += RG_WARPS * 32 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.rn + i));
  pdl_wait();
  pdl_launch_dependents();
  float sq = rg_stage(p, xs);
  if (p.res) sq = rg_residual(p, xs, sq, red);
  if (p.nw) rg_norm(p, xs, sq, red);
  __syncthreads();
  float acc[R][2];
#pragma unroll
  for (int r = 0; r < R; r++) acc[r][0] = acc[r][1] = 0.f;
  while (rg < groups) {
    int ng = rg, nb = cb + 32 * U;
    if (nb >= c_hi) { ng += stride; nb = c_lo; }
    if (ng < groups) fetch(nxt, ng, nb);
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int c = cb + lane + 32 * u;
      if (c < c_hi) {
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
        if (ks == 1) {
          rg_emit<R>(p, rg, a);
        } else {
#pragma unroll
          for (int r = 0; r < R; r++) part[((loc * ns + stream) * R + r) * ks + sub] = a[r];
        }
      }
      loc++;
    }
    rg = ng;
    cb = nb;
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
      for (int u = 0; u < U; u++) cur[r][u] = nxt[r][u];
  }
  if (ks == 1) return;
  __syncthreads();
  for (int i = tid;; i += RG_WARPS * 32) {
    const int l = i / ns, g = (blockIdx.x * ns + i - l * ns) + l * stride;
    if (l * stride + (int)blockIdx.x * ns >= groups) break;
    if (g >= groups) continue;
    float a[R];
#pragma unroll
    for (int r = 0; r < R; r++) {
      a[r] = 0.f;
      for (int k = 0; k < ks; k++) a[r] += part[(i * R + r) * ks + k];
    }
    rg_emit<R>(p, g, a);
  }
}

template <typename WT, int R>
int rg_launch(DeviceCtx* c, const RowGemv& p, cudaStream_t s) {
  static std::atomic<unsigned long long> done{0};
  const int rc = ensure_dynamic_smem(row_gemv_kernel<WT, R>, 220 * 1024, done);
  if (rc) return rc;
  const int groups = (p.N + R - 1) / R, chunks = (int)(p.ldw / Vec16<WT>::N), full = 2 * c->sm_count;
  // warps a stream (single rows): the fewest that come within 3 % of the most even division
  int ks = 1;
  double best = 1e30;
  for (int k = 1; k <= RG_WARPS; k *= 2) {
    if (k > 1 && chunks / k < 32 * 4) break;
    const int ns = RG_WARPS / k;
    const double cost = (double)((groups + full * ns - 1) / (full * ns)) / k;
    if (cost < best * 0.97) { best = cost; ks = k; }
    if (R == 2) break;   // two rows a warp: the extra sums cost more than the unevenness
  }
  const int ns = RG_WARPS / ks, need = (groups + ns - 1) / ns, ctas = need < full ? need : full;
  const int local = (groups + ctas * ns - 1) / (ctas * ns);
  const size_t smem = ((size_t)p.ldw + (ks > 1 ? (size_t)local * ns * R * ks : 0)) * sizeof(float);
  if (smem > 220 * 1024) return set_error(TLB_ERR_UNSUPPORTED, "row_gemv: the activation row does not fit the shared-memory stage");
  LaunchCfg lc(dim3(ctas), dim3(RG_WARPS * 32), smem, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, row_gemv_kernel<WT, R>, p, ks));
  return TLB_OK;
}

// ---- row ops of the prompt pass --------------------------------------------------------------
template <typename OT>
__global__ void __launch_bounds__(256) rms_rows_kernel(const float* __restrict__ x, long long ldx,
                                                       const float* __restrict__ w, OT* __restrict__ out, long long ldo,
                                                       int n, float eps, float scale) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const float* row = x + (size_t)blockIdx.x * ldx;
  OT* dst = out + (size_t)blockIdx.x * ldo;
  float sq = 0.f;
  for (int i = threadIdx.x; i < n; i += 256) sq = fmaf(row[i], row[i], sq);
  sq = block_sum(sq, red);
  const float r = rsqrtf(sq / n + eps) * scale;
  for (int i = threadIdx.x; i < n; i += 256) put(dst + i, row[i] * r * w[i]);
}

// x += norm(y) * w, the sum also as the next product's operand; without y only the latter
constexpr int RR_HOLD = 8;    // values of y a thread keeps between the passes
template <typename OT>
__global__ void __launch_bounds__(512) residual_rows_kernel(float* __restrict__ x, const float* __restrict__ y,
                                                            const float* __restrict__ w, OT* __restrict__ out,
                                                            long long ldo, int n, float eps) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  float* row = x + (size_t)blockIdx.x * n;
  OT* dst = out + (size_t)blockIdx.x * ldo;
  if (!y) {
    for (int i = threadIdx.x; i < n; i += 512) put(dst + i, row[i]);
    return;
  }
  const float* yr = y + (size_t)blockIdx.x * n;
  float v[RR_HOLD], sq = 0.f;
#pragma unroll
  for (int k = 0; k < RR_HOLD; k++) {
    const int i = threadIdx.x + k * 512;
    v[k] = i < n ? yr[i] : 0.f;
    sq = fmaf(v[k], v[k], sq);
  }
  for (int i = threadIdx.x + RR_HOLD * 512; i < n; i += 512) sq = fmaf(yr[i], yr[i], sq);
  sq = block_sum(sq, red);
  const float r = rsqrtf(sq / n + eps);
#pragma unroll
  for (int k = 0; k < RR_HOLD; k++) {
    const int i = threadIdx.x + k * 512;
    if (i < n) {
      const float s = fmaf(v[k] * r, w[i], row[i]);
      row[i] = s;
      put(dst + i, s);
    }
  }
  for (int i = threadIdx.x + RR_HOLD * 512; i < n; i += 512) {
    const float s = fmaf(yr[i] * r, w[i], row[i]);
    row[i] = s;
    put(dst + i, s);
  }
}

// 1024 columns a block
template <typename WT>
__global__ void embed_scaled_kernel(const WT* __restrict__ embed, long long ld, const int* __restrict__ ids,
                                    float* __restrict__ x, int width, float scale) {
  pdl_wait();
  pdl_launch_dependents();
  const WT* src = embed + (size_t)ids[blockIdx.x] * ld;
#pragma unroll
  for (int k = 0; k < 4; k++) {
    const int i = blockIdx.y * 1024 + k * 256 + threadIdx.x;
    if (i < width) x[(size_t)blockIdx.x * width + i] = to_f(src[i]) * scale;
  }
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

__global__ void relu2_rows_kernel(const float* __restrict__ u, float* __restrict__ out, long long n) {
  pdl_wait();
  pdl_launch_dependents();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
    out[i] = relu2(u[i]);
}

}  // namespace

int row_gemv_launch(DeviceCtx* c, const RowGemv& p, bool bf16, cudaStream_t s) {
  // two rows a stream where the rows come in pairs, or where there are enough of them to fill the SMs
  const bool two = p.epi == 2 || p.N >= 2 * 2 * c->sm_count * RG_WARPS;
  if (bf16) return two ? rg_launch<__nv_bfloat16, 2>(c, p, s) : rg_launch<__nv_bfloat16, 1>(c, p, s);
  return two ? rg_launch<float, 2>(c, p, s) : rg_launch<float, 1>(c, p, s);
}

int rms_rows_launch(const float* x, long long ldx, const float* w, void* out, long long ldo, int n, float eps,
                    float scale, int rows, bool bf16, cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(256), 0, s, pdl_enabled());
  if (bf16)
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, rms_rows_kernel<__nv_bfloat16>, x, ldx, w, (__nv_bfloat16*)out, ldo, n, eps, scale));
  else
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, rms_rows_kernel<float>, x, ldx, w, (float*)out, ldo, n, eps, scale));
  return TLB_OK;
}

int residual_rows_launch(float* x, const float* y, const float* w, void* out, long long ldo, int n, float eps, int rows,
                         bool bf16, cudaStream_t s) {
  LaunchCfg lc(dim3(rows), dim3(512), 0, s, pdl_enabled());
  if (bf16)
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, residual_rows_kernel<__nv_bfloat16>, x, y, w, (__nv_bfloat16*)out, ldo, n, eps));
  else
    TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, residual_rows_kernel<float>, x, y, w, (float*)out, ldo, n, eps));
  return TLB_OK;
}

int relu2_rows_launch(const float* u, float* out, int ff, int rows, cudaStream_t s) {
  const long long n = (long long)rows * ff, b = (n + 255) / 256;
  LaunchCfg lc(dim3((unsigned)(b < 148 * 16 ? b : 148 * 16)), dim3(256), 0, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, relu2_rows_kernel, u, out, n));
  return TLB_OK;
}

int embed_scaled_launch(const void* embed, const int* ids, float* x, int width, long long ld, float scale, int rows,
                        bool bf16, cudaStream_t s) {
  LaunchCfg lc(dim3(rows, (width + 1023) / 1024), dim3(256), 0, s, pdl_enabled());
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
