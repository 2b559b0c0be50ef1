// Activation applied to a product's fp32 accumulators before they are stored (GEMV, tcgen05 GEMM and FP32-unit GEMM share it).
//   1  squared relu
//   2  gelu_tanh(v) * table[ids[row]][off + col]: a row of an embedding table gated by the product (columns from `n` on, and
//      ids outside the table, give 0)
//   3  v * sigmoid(table[ids ? ids[row] : row][off + col]): a gate per element, columns counted over the heads of a batched product
// And the gated activation of a [gate | up] pair.
#pragma once
#include "rows.cuh"

namespace spark {

struct OutAct {
  int kind;
  int ld, off, n, rows, f32;        // the table: row stride, first column, valid columns, rows, element type
  const void* table;
  const int* ids;
  int batch_cols;                   // columns per item of a batched product: `col` is item * batch_cols + the item's column
};

// g sigmoid(alpha g) (u + shift); with a limit > 0, g is at most the limit and u within +- the limit before that.
struct GluAct { float limit, alpha, shift; };

template <typename T>
__device__ __forceinline__ float glu_t(const GluAct& a, float g, float u) {
  if (a.limit > 0.f) { g = fminf(g, a.limit); u = fminf(fmaxf(u, -a.limit), a.limit); }
  const float z = a.alpha * g;
  const float s = sizeof(T) == 2 ? __fdividef(g, 1.f + __expf(-z)) : g / (1.f + expf(-z));
  return s * (u + a.shift);
}

__device__ __forceinline__ float relu2_f(float v) { v = fmaxf(v, 0.f); return v * v; }

__device__ __forceinline__ float out_act(const OutAct& a, float v, int row, int col) {
  if (a.kind == 0) return v;
  if (a.kind == 1) return relu2_f(v);
  if (a.kind == 3) {
    const size_t i = static_cast<size_t>(a.ids ? a.ids[row] : row) * a.ld + a.off + col;
    return v * (a.f32 ? sigmoid_f(static_cast<const float*>(a.table)[i])
                      : sigmoid_t<__nv_bfloat16>(__bfloat162float(static_cast<const __nv_bfloat16*>(a.table)[i])));
  }
  const int id = a.ids[row];
  if (col >= a.n || id < 0 || id >= a.rows) return 0.f;
  const size_t i = static_cast<size_t>(id) * a.ld + a.off + col;
  const float e = a.f32 ? static_cast<const float*>(a.table)[i] : __bfloat162float(static_cast<const __nv_bfloat16*>(a.table)[i]);
  return gelu_tanh_f(v) * e;
}

}  // namespace spark
