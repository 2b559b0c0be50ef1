// Batched C[b] = A[b] B[b]^T on the FP32 units (64 x 64 tiles, 4 x 4 per thread): the product of the 32-bit mode (no
// reduced-precision matrix mode anywhere), and of bf16 shapes that the TMA / vector kernels cannot address (a
// contraction length or row stride that is not a multiple of 8).  The grouped form walks the tile list of the expert sort.
#include "../common/out_act.cuh"

namespace spark {

// grouped: tiles of <= 128 rows {first row, end of the expert's rows, expert, 0} in expert order; A row of a sorted row p is
// perm[p] / a_div (perm null: p); B starts at expert * sb, C rows are sorted rows.
struct SimtGroups { const int4* tiles; const int* count; const int* perm; int a_div; };

template <typename T, typename TC>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, int lda, long long sa, const T* __restrict__ B, int ldb, long long sb, TC* __restrict__ C,
                 int ldc, long long sc, int M, int N, int K, OutAct act, SimtGroups grp) {
  __shared__ float As[16][68], Bs[16][68];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  int m0 = blockIdx.y * 64;
  const int n0 = blockIdx.x * 64;
  if (grp.tiles) {
    if (static_cast<int>(blockIdx.y >> 1) >= *grp.count) return;
    const int4 tl = grp.tiles[blockIdx.y >> 1];
    m0 = tl.x + (blockIdx.y & 1) * 64;
    M = min(tl.y, tl.x + 128);
    if (m0 >= M) return;
    B += tl.z * sb;
  } else {
    A += blockIdx.z * sa; B += blockIdx.z * sb; C += blockIdx.z * sc;
  }
  const int lr = tid >> 4, lk = tid & 15;                    // rows lr, lr + 16, ... of both operands, one k each
  const T* ar[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    int r = min(m0 + lr + 16 * i, M - 1);
    if (grp.perm) r = grp.perm[r] / grp.a_div;
    ar[i] = A + static_cast<size_t>(r) * lda;
  }
  const int oc = grp.tiles ? 0 : blockIdx.z * act.batch_cols;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i, k = k0 + lk;
      As[lk][r] = (m0 + r < M && k < K) ? ldf(ar[i] + k) : 0.f;
      Bs[lk][r] = (n0 + r < N && k < K) ? ldf(B + static_cast<size_t>(n0 + r) * ldb + k) : 0.f;
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
      if (m < M && n < N) stf(C + static_cast<size_t>(m) * ldc + n, out_act(act, acc[i][j], m, oc + n));
    }
}

}  // namespace spark

using namespace spark;

#define SPARK_SIMT(grid)                                                                                                              \
  if (f32_in) gemm_simt_kernel<float, float><<<grid, 256, 0, s>>>((const float*)A, lda, sa, (const float*)B, ldb, sb, (float*)C, ldc, \
                                                                  sc, M, N, K, a, grp);                                               \
  else if (f32_out) gemm_simt_kernel<__nv_bfloat16, float><<<grid, 256, 0, s>>>((const __nv_bfloat16*)A, lda, sa,                     \
                                                                                (const __nv_bfloat16*)B, ldb, sb, (float*)C, ldc, sc, \
                                                                                M, N, K, a, grp);                                     \
  else gemm_simt_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, 256, 0, s>>>((const __nv_bfloat16*)A, lda, sa,                          \
                                                                           (const __nv_bfloat16*)B, ldb, sb, (__nv_bfloat16*)C, ldc,  \
                                                                           sc, M, N, K, a, grp);

// f32_in: fp32 A and B (C fp32); else bf16 A and B with C bf16 or fp32 (f32_out).  Strides in elements.  act: optional (host).
extern "C" int spark_gemm_simt(const void* A, int lda, long long sa, const void* B, int ldb, long long sb, void* C, int ldc,
                               long long sc, int batch, int M, int N, int K, int f32_in, int f32_out, const OutAct* act,
                               cudaStream_t s) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if ((M + 63) / 64 > 65535 || batch > 65535) return -5;
  const dim3 grid((N + 63) / 64, (M + 63) / 64, batch);
  const OutAct a = act ? *act : OutAct{};
  const SimtGroups grp{};
  SPARK_SIMT(grid)
  return spark_launch_rc(__func__);
}

// Grouped over a device-side tile list (see spark_moe_sort); perm / a_div: rows of A by sorted row (perm null: A is sorted).
extern "C" int spark_gemm_simt_grouped(const void* A, int lda, const void* B, int ldb, long long sb, void* C, int ldc, int N, int K,
                                       const void* tiles, const int* count, int max_tiles, const int* perm, int a_div, int f32_in,
                                       int f32_out, const OutAct* act, cudaStream_t s) {
  if (max_tiles <= 0 || N <= 0) return 0;
  if (2 * max_tiles > 65535) return -5;
  const dim3 grid((N + 63) / 64, 2 * max_tiles, 1);
  const OutAct a = act ? *act : OutAct{};
  const SimtGroups grp{(const int4*)tiles, count, perm, a_div};
  const long long sa = 0, sc = 0;
  const int M = 0;
  SPARK_SIMT(grid)
  return spark_launch_rc(__func__);
}
