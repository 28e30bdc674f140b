// bf16 matrix product of a prompt pass: C[M,N] = A[M,K] . W[N,K]^T on the 5th-generation tensor
// cores, f32 accumulation, with what follows the product done in its epilogue:
//   EPI 0  C[m,n]  = acc                      (f32)
//   EPI 1  C[m,n] += acc                      (f32 residual)
//   EPI 2  O[m,j]  = glu(acc[2j], acc[2j+1])  (bf16, gate and up rows interleaved in W)
//   EPI 3  O[m,n]  = acc                      (bf16)
//   EPI 4  O[m,n]  = relu(acc)^2              (bf16)
//
// Persistent: one CTA per SM walks the 128 x BN output tiles.  Warp 0 is the TMA producer of both
// operands (64-k stages, 128-byte swizzle, boxes past M, N or K read as zeros), warp 1 issues
// tcgen05.mma (the whole warp runs the loop, one elected lane issues), warps 4-7 read the
// accumulator back with tcgen05.ld and store.  Two TMEM accumulators in rotation, so the epilogue
// of a tile runs under the products of the next.  BN (32 / 64 / 128 / 256) is picked on the host so
// that short prompts still occupy the SMs.  All waits are bounded: a timeout sets the status word,
// the kernel frees its TMEM and returns.  No cluster launch, no multicast.
#include <cuda_bf16.h>

#include "common.cuh"
#include "mixers.cuh"

namespace tlb {

namespace {

constexpr int GT_THREADS = 256;
constexpr int GT_M = 128;   // activation rows per tile (UMMA M)
constexpr int GT_KS = 64;   // k per stage: one 128-byte swizzle row of bf16

struct GtParams {
  float* C;
  long long ldc;
  __nv_bfloat16* O;
  long long ldo;
  int M, N, K;
  int mt, nt;        // tiles along M and N
  float limit;
  int* status;
};

template <int BN>
struct GtSmem {
  static constexpr int STAGES = BN == 256 ? 4 : (BN == 128 ? 6 : 8);
  static constexpr size_t A = 0;
  static constexpr size_t B = A + (size_t)STAGES * GT_M * 128;
  static constexpr size_t BARS = B + (size_t)STAGES * BN * 128;
  static constexpr size_t SLOT = BARS + (2 * STAGES + 4) * 8;
  static constexpr size_t TOTAL = SLOT + 16 + 1024;
};

__device__ __forceinline__ void gt_mma(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d),
      "l"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ void gt_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void gt_ld32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
      "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];\n\t"
      "tcgen05.wait::ld.sync.aligned;"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
        "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]),
        "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
// K-major operand with 128-byte swizzle: rows of 128 bytes, 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t gt_desc(uint32_t addr) {
  return (uint64_t)((addr & 0x3FFFFu) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) |
         ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}
// kind::f16, both operands bf16 and K-major, f32 accumulate, M = 128, N = n
__device__ __forceinline__ uint32_t gt_idesc(int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(GT_M >> 4) << 24);
}
__device__ __forceinline__ bool gt_wait_warp(uint64_t* bar, uint32_t parity, int* status, int where) {
  return __all_sync(0xffffffffu, mbar_wait_bounded(bar, parity, status, where));
}

template <int BN, int EPI>
__global__ void __launch_bounds__(GT_THREADS, 1)
    gemm_bf16_tc_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, GtParams p) {
  using S = GtSmem<BN>;
  constexpr int ST = S::STAGES;
  constexpr uint32_t NCOLS = 2 * BN < 32 ? 32 : 2 * BN;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* base = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  uint64_t* full = (uint64_t*)(base + S::BARS);
  uint64_t* empty = full + ST;
  uint64_t* dfull = empty + ST;
  uint64_t* dempty = dfull + 2;
  uint32_t* slot = (uint32_t*)(base + S::SLOT);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nk = (p.K + GT_KS - 1) / GT_KS, tiles = p.mt * p.nt;

  if (tid == 0) {
    for (int s = 0; s < ST; s++) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    for (int b = 0; b < 2; b++) { mbar_init(&dfull[b], 1); mbar_init(&dempty[b], 4); }
    mbar_fence_init();
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(slot)), "r"(NCOLS)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *slot;
  pdl_wait();
  pdl_launch_dependents();

  if (warp == 0) {
    if (lane == 0) {
      int it = 0;
      bool ok = true;
      for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
        const int m0 = (t % p.mt) * GT_M, n0 = (t / p.mt) * BN;
        for (int k = 0; k < nk; k++, it++) {
          const int s = it % ST;
          if (!mbar_wait_bounded(&empty[s], ((it / ST) & 1) ^ 1, p.status, 700)) { ok = false; break; }
          mbar_expect_tx(&full[s], (uint32_t)(GT_M + BN) * 128u);
          tma_load_2d(base + S::A + (size_t)s * GT_M * 128, &tmA, k * GT_KS, m0, &full[s]);
          tma_load_2d(base + S::B + (size_t)s * BN * 128, &tmB, k * GT_KS, n0, &full[s]);
        }
      }
    }
  } else if (warp == 1) {
    const uint32_t idesc = gt_idesc(BN);
    uint32_t pred;
    asm volatile("{\n\t.reg .pred p;\n\telect.sync _|p, 0xffffffff;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(pred));
    const bool leader = pred != 0;
    int it = 0, n = 0;
    bool ok = true;
    for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, n++) {
      const int buf = n & 1;
      if (!gt_wait_warp(&dempty[buf], ((n >> 1) & 1) ^ 1, p.status, 711)) break;
      const uint32_t d = tmem + (uint32_t)(buf * BN);
      for (int k = 0; k < nk; k++, it++) {
        const int s = it % ST;
        if (!gt_wait_warp(&full[s], (it / ST) & 1, p.status, 710)) { ok = false; break; }
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint64_t a = gt_desc(smem_u32(base + S::A + (size_t)s * GT_M * 128));
        const uint64_t b = gt_desc(smem_u32(base + S::B + (size_t)s * BN * 128));
        if (leader) {
#pragma unroll
          for (int ks = 0; ks < GT_KS / 16; ks++)
            gt_mma(d, a + (uint64_t)(ks * 2), b + (uint64_t)(ks * 2), idesc, (k | ks) ? 1u : 0u);
          gt_commit(&empty[s]);
          if (k + 1 == nk) gt_commit(&dfull[buf]);
        }
        __syncwarp();
      }
    }
  } else if (warp >= 4) {
    const int quarter = warp & 3;
    int n = 0;
    for (int t = blockIdx.x; t < tiles; t += gridDim.x, n++) {
      const int buf = n & 1;
      const int m = (t % p.mt) * GT_M + quarter * 32 + lane, n0 = (t / p.mt) * BN;
      if (!gt_wait_warp(&dfull[buf], (n >> 1) & 1, p.status, 720)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t taddr = tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(buf * BN);
#pragma unroll 1
      for (int c0 = 0; c0 < BN; c0 += 32) {
        uint32_t v[32];
        gt_ld32(taddr + (uint32_t)c0, v);
        if (c0 + 32 >= BN) {
          asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
          __syncwarp();
          if (lane == 0) mbar_arrive(&dempty[buf]);
        }
        if (m >= p.M) continue;
        if (EPI == 2) {
          __nv_bfloat16* o = p.O + (long long)m * p.ldo + (n0 + c0) / 2;
          if (n0 + c0 + 32 <= p.N && (p.ldo & 7) == 0) {
            uint32_t w[8];
#pragma unroll
            for (int j = 0; j < 8; j++) {
              const __nv_bfloat162 h = __floats2bfloat162_rn(
                  glu_clipped(__uint_as_float(v[4 * j]), __uint_as_float(v[4 * j + 1]), p.limit),
                  glu_clipped(__uint_as_float(v[4 * j + 2]), __uint_as_float(v[4 * j + 3]), p.limit));
              w[j] = *(const uint32_t*)&h;
            }
            ((uint4*)o)[0] = make_uint4(w[0], w[1], w[2], w[3]);
            ((uint4*)o)[1] = make_uint4(w[4], w[5], w[6], w[7]);
          } else {
#pragma unroll
            for (int j = 0; j < 16; j++)
              if (n0 + c0 + 2 * j + 1 < p.N)
                o[j] = __float2bfloat16_rn(
                    glu_clipped(__uint_as_float(v[2 * j]), __uint_as_float(v[2 * j + 1]), p.limit));
          }
        } else if (EPI >= 3) {
          __nv_bfloat16* o = p.O + (long long)m * p.ldo + n0 + c0;
          if (EPI == 4) {
#pragma unroll
            for (int j = 0; j < 32; j++) v[j] = __float_as_uint(relu2(__uint_as_float(v[j])));
          }
          if (n0 + c0 + 32 <= p.N && (p.ldo & 7) == 0) {
#pragma unroll
            for (int j = 0; j < 4; j++) {
              uint32_t w[4];
#pragma unroll
              for (int k = 0; k < 4; k++) {
                const __nv_bfloat162 h = __floats2bfloat162_rn(__uint_as_float(v[8 * j + 2 * k]), __uint_as_float(v[8 * j + 2 * k + 1]));
                w[k] = *(const uint32_t*)&h;
              }
              ((uint4*)o)[j] = make_uint4(w[0], w[1], w[2], w[3]);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; j++)
              if (n0 + c0 + j < p.N) o[j] = __float2bfloat16_rn(__uint_as_float(v[j]));
          }
        } else {
          float* o = p.C + (long long)m * p.ldc + n0 + c0;
          if (n0 + c0 + 32 <= p.N && (p.ldc & 3) == 0) {
#pragma unroll
            for (int j = 0; j < 8; j++) {
              float4 f = make_float4(__uint_as_float(v[4 * j]), __uint_as_float(v[4 * j + 1]),
                                     __uint_as_float(v[4 * j + 2]), __uint_as_float(v[4 * j + 3]));
              if (EPI == 1) {
                const float4 r = ((const float4*)o)[j];
                f.x += r.x; f.y += r.y; f.z += r.z; f.w += r.w;
              }
              ((float4*)o)[j] = f;
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; j++)
              if (n0 + c0 + j < p.N) o[j] = __uint_as_float(v[j]) + (EPI == 1 ? o[j] : 0.f);
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(NCOLS) : "memory");
  }
}

int encode_operand(EncodeTiledFn enc, CUtensorMap* tm, const void* p, int rows, int K, long long ld, int box_rows) {
  cuuint64_t dim[2] = {(cuuint64_t)K, (cuuint64_t)rows};
  cuuint64_t str[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {(cuuint32_t)GT_KS, (cuuint32_t)box_rows};
  cuuint32_t es[2] = {1, 1};
  if (enc(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p), dim, str, box, es,
          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return set_error(TLB_ERR_CUDA, "gemm_bf16_tc: tensor map encode failed");
  return TLB_OK;
}

template <int BN, int EPI>
int gt_launch(DeviceCtx* c, const CUtensorMap& ta, const CUtensorMap& tb, const GtParams& p, cudaStream_t s) {
  static std::atomic<unsigned long long> attr_done{0};
  {
    const int rc = ensure_dynamic_smem(gemm_bf16_tc_kernel<BN, EPI>, (int)GtSmem<BN>::TOTAL, attr_done);
    if (rc) return rc;
  }
  const int tiles = p.mt * p.nt;
  LaunchCfg lc(dim3(tiles < c->sm_count ? tiles : c->sm_count), dim3(GT_THREADS), GtSmem<BN>::TOTAL, s, pdl_enabled());
  TLB_CUDA(cudaLaunchKernelEx(&lc.cfg, gemm_bf16_tc_kernel<BN, EPI>, ta, tb, p));
  return TLB_OK;
}

}  // namespace

bool gemm_bf16_tc_eligible(const void* a, long long lda, const void* w, long long ldw) {
  return lda % 8 == 0 && ldw % 8 == 0 && ((uintptr_t)a & 15) == 0 && ((uintptr_t)w & 15) == 0;
}

int gemm_bf16_tc_launch(DeviceCtx* c, const void* a, long long lda, const void* w, long long ldw, float* C,
                        long long ldc, void* O, long long ldo, int M, int N, int K, int epi, float limit,
                        cudaStream_t s) {
  EncodeTiledFn enc = encode_tiled_fn();
  if (!enc) return set_error(TLB_ERR_CUDA, "cuTensorMapEncodeTiled entry point not found");
  if (!gemm_bf16_tc_eligible(a, lda, w, ldw) || M <= 0 || N <= 0 || K <= 0)
    return set_error(TLB_ERR_ARG, "gemm_bf16_tc: operands must be 16-byte aligned with row strides of 8 elements");
  const int mt = (M + GT_M - 1) / GT_M;
  // widest tile that still gives every SM work
  int BN = 256;
  while (BN > 32 && mt * ((N + BN - 1) / BN) < c->sm_count) BN >>= 1;
  CUtensorMap ta, tb;
  int rc = encode_operand(enc, &ta, a, M, K, lda, GT_M);
  if (!rc) rc = encode_operand(enc, &tb, w, N, K, ldw, BN);
  if (rc) return rc;
  GtParams p{C, ldc, (__nv_bfloat16*)O, ldo, M, N, K, mt, (N + BN - 1) / BN, limit, c->status};
#define GT_CASE(bn)                                                            \
  if (BN == bn) switch (epi) {                                                 \
      case 0: return gt_launch<bn, 0>(c, ta, tb, p, s);                        \
      case 1: return gt_launch<bn, 1>(c, ta, tb, p, s);                        \
      case 2: return gt_launch<bn, 2>(c, ta, tb, p, s);                        \
      case 3: return gt_launch<bn, 3>(c, ta, tb, p, s);                        \
      default: return gt_launch<bn, 4>(c, ta, tb, p, s);                       \
    }
  GT_CASE(256) GT_CASE(128) GT_CASE(64) GT_CASE(32)
#undef GT_CASE
  return set_error(TLB_ERR_STATE, "gemm_bf16_tc: no tile width");
}

}  // namespace tlb
