// C = A * B^T on the CUDA cores, fp32 accumulation in one fixed K order per element (a row's result does not depend on
// the rest of the batch). Two uses: the engine's full-precision mode (fp32 operands: the tensor cores would round them),
// and bf16 operands whose row pitch a TMA descriptor cannot describe. A [M, K], B [N, K], C [M, N], all row-major.
// tile_boff (grouped form, one int per 128 rows of A): first row of B of that tile's expert.
// sb_gemm_simt_heads: one product per head z, C[:, z] = A[:, z] * B[z]^T with B stored [N, K] or [K, N] (b_kn), times sigmoid(gate).
#include "common.cuh"

namespace sb {

constexpr int SG_BM = 64, SG_BN = 64, SG_BK = 16;

__device__ __forceinline__ float sg_load(const float* p) { return *p; }
__device__ __forceinline__ float sg_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void sg_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void sg_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <typename T, typename TO>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ B, TO* __restrict__ C, const T* __restrict__ bias,
                 const int* __restrict__ tile_boff, int M, int N, int K, long lda, long ldb, long ldc) {
  __shared__ float sA[SG_BK][SG_BM + 4], sB[SG_BK][SG_BN + 4];
  pdl_wait();
  pdl_launch_dependents();
  const int m0 = blockIdx.y * SG_BM, n0 = blockIdx.x * SG_BN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* b = B + (tile_boff != nullptr ? static_cast<long>(tile_boff[m0 / 128]) * ldb : 0);
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SG_BK) {
    for (int i = threadIdx.x; i < SG_BM * SG_BK; i += 256) {
      const int r = i / SG_BK, c = i % SG_BK;
      sA[c][r] = (m0 + r < M && k0 + c < K) ? sg_load(A + (m0 + r) * lda + k0 + c) : 0.f;
      sB[c][r] = (n0 + r < N && k0 + c < K) ? sg_load(b + (n0 + r) * ldb + k0 + c) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_BK; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        x[i] = sA[k][ty * 4 + i];
        y[i] = sB[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) sg_store(C + m * ldc + n, acc[i][j] + (bias != nullptr ? sg_load(bias + n) : 0.f));
    }
  }
}

struct HeadGemm {
  int M, N, K, b_kn;
  long a_row, a_head, b_head, b_ld, c_row, c_head, gate_row, gate_head;  // elements
};

template <typename T>
__global__ void __launch_bounds__(256)
gemm_simt_heads_kernel(const T* __restrict__ A, const T* __restrict__ B, T* __restrict__ C, const T* __restrict__ gate,
                       const __grid_constant__ HeadGemm g) {
  __shared__ float sA[SG_BK][SG_BM + 4], sB[SG_BK][SG_BN + 4];
  pdl_wait();
  pdl_launch_dependents();
  const int n0 = blockIdx.x * SG_BN, m0 = blockIdx.y * SG_BM, z = blockIdx.z;
  const T* a = A + z * g.a_head;
  const T* b = B + z * g.b_head;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.K; k0 += SG_BK) {
    for (int i = threadIdx.x; i < SG_BM * SG_BK; i += 256) {
      const int r = i / SG_BK, c = i % SG_BK;
      sA[c][r] = (m0 + r < g.M && k0 + c < g.K) ? sg_load(a + (m0 + r) * g.a_row + k0 + c) : 0.f;
      // the stored order decides which index runs fastest, so that neighbouring threads read neighbouring elements
      const int bn = g.b_kn ? i % SG_BN : r, bk = g.b_kn ? i / SG_BN : c;
      sB[bk][bn] = (n0 + bn < g.N && k0 + bk < g.K) ? sg_load(g.b_kn ? b + (k0 + bk) * g.b_ld + n0 + bn : b + (n0 + bn) * g.b_ld + k0 + bk) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_BK; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        x[i] = sA[k][ty * 4 + i];
        y[i] = sB[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= g.M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= g.N) continue;
      const float f = gate != nullptr ? 1.f / (1.f + expf(-sg_load(gate + m * g.gate_row + z * g.gate_head + n))) : 1.f;
      sg_store(C + m * g.c_row + z * g.c_head + n, acc[i][j] * f);
    }
  }
}

}  // namespace sb

extern "C" int sb_gemm_simt_heads(const void* A, const void* B, void* C, const void* gate, int H, int M, int N, int K, int b_kn, long a_row,
                                  long a_head, long b_head, long b_ld, long c_row, long c_head, long gate_row, long gate_head, int f32,
                                  cudaStream_t s) {
  if (H <= 0 || M <= 0 || N <= 0) return 0;
  if (H > 65535 || (M + sb::SG_BM - 1) / sb::SG_BM > 65535) return (int)cudaErrorInvalidValue;
  const dim3 grid((N + sb::SG_BN - 1) / sb::SG_BN, (M + sb::SG_BM - 1) / sb::SG_BM, H);
  const sb::HeadGemm g{M, N, K, b_kn, a_row, a_head, b_head, b_ld, c_row, c_head, gate_row, gate_head};
  using bf16 = __nv_bfloat16;
  if (f32)
    return (int)sb::launch_pdl(sb::gemm_simt_heads_kernel<float>, grid, dim3(256), 0, s, (const float*)A, (const float*)B, (float*)C,
                               (const float*)gate, g);
  return (int)sb::launch_pdl(sb::gemm_simt_heads_kernel<bf16>, grid, dim3(256), 0, s, (const bf16*)A, (const bf16*)B, (bf16*)C,
                             (const bf16*)gate, g);
}

extern "C" int sb_gemm_simt(const void* A, const void* B, void* C, const void* bias, const int* tile_boff, int M, int N, int K,
                            long lda, long ldb, long ldc, int in_f32, int out_f32, cudaStream_t s) {
  if (M <= 0 || N <= 0) return 0;
  if ((M + sb::SG_BM - 1) / sb::SG_BM > 65535) return (int)cudaErrorInvalidValue;
  const dim3 grid((N + sb::SG_BN - 1) / sb::SG_BN, (M + sb::SG_BM - 1) / sb::SG_BM);
  using bf16 = __nv_bfloat16;
  if (in_f32 && !out_f32) return (int)cudaErrorInvalidValue;
  if (in_f32)
    return (int)sb::launch_pdl(sb::gemm_simt_kernel<float, float>, grid, dim3(256), 0, s, (const float*)A, (const float*)B, (float*)C,
                               (const float*)bias, tile_boff, M, N, K, lda, ldb, ldc);
  if (out_f32)
    return (int)sb::launch_pdl(sb::gemm_simt_kernel<bf16, float>, grid, dim3(256), 0, s, (const bf16*)A, (const bf16*)B, (float*)C,
                               (const bf16*)bias, tile_boff, M, N, K, lda, ldb, ldc);
  return (int)sb::launch_pdl(sb::gemm_simt_kernel<bf16, bf16>, grid, dim3(256), 0, s, (const bf16*)A, (const bf16*)B, (bf16*)C,
                             (const bf16*)bias, tile_boff, M, N, K, lda, ldb, ldc);
}
