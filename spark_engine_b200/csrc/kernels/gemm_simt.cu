// Batched C[b] = A[b] B[b]^T on the FP32 units (64 x 64 tiles, 4 x 4 per thread): the product of the 32-bit mode (no
// reduced-precision matrix mode anywhere), and of bf16 shapes that the TMA / vector kernels cannot address (a
// contraction length or row stride that is not a multiple of 8).
#include "../common/rows.cuh"

namespace spark {

template <typename T, typename TC>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, int lda, long long sa, const T* __restrict__ B, int ldb, long long sb, TC* __restrict__ C,
                 int ldc, long long sc, int M, int N, int K) {
  __shared__ float As[16][68], Bs[16][68];
  A += blockIdx.z * sa; B += blockIdx.z * sb; C += blockIdx.z * sc;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = tid; i < 1024; i += 256) {
      const int r = i >> 4, k = i & 15;
      As[k][r] = (m0 + r < M && k0 + k < K) ? ldf(A + static_cast<size_t>(m0 + r) * lda + k0 + k) : 0.f;
      Bs[k][r] = (n0 + r < N && k0 + k < K) ? ldf(B + static_cast<size_t>(n0 + r) * ldb + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&As[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) stf(C + static_cast<size_t>(m) * ldc + n, acc[i][j]);
    }
}

}  // namespace spark

using namespace spark;

// f32_in: fp32 A and B (C fp32); else bf16 A and B with C bf16 or fp32 (f32_out).  Strides in elements.
extern "C" int spark_gemm_simt(const void* A, int lda, long long sa, const void* B, int ldb, long long sb, void* C, int ldc,
                               long long sc, int batch, int M, int N, int K, int f32_in, int f32_out, cudaStream_t s) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if ((M + 63) / 64 > 65535 || batch > 65535) return -5;
  const dim3 grid((N + 63) / 64, (M + 63) / 64, batch);
  if (f32_in) gemm_simt_kernel<float, float><<<grid, 256, 0, s>>>((const float*)A, lda, sa, (const float*)B, ldb, sb, (float*)C, ldc, sc, M, N, K);
  else if (f32_out) gemm_simt_kernel<__nv_bfloat16, float><<<grid, 256, 0, s>>>((const __nv_bfloat16*)A, lda, sa, (const __nv_bfloat16*)B, ldb, sb, (float*)C, ldc, sc, M, N, K);
  else gemm_simt_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, 256, 0, s>>>((const __nv_bfloat16*)A, lda, sa, (const __nv_bfloat16*)B, ldb, sb, (__nv_bfloat16*)C, ldc, sc, M, N, K);
  return spark_launch_rc(__func__);
}
