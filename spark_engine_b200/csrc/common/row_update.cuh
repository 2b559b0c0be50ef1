// Update of the residual stream and the norm of its rows: arguments shared by the row kernels.
#pragma once
#include "rows.cuh"

namespace spark {

struct RowUpdate {
  float* res;                                   // [R, H]
  // the update: `delta` rows, or sum over slots of wts (null: 1) * y (expert outputs) + sg * shared + self_w * self_x, or nothing
  const float* delta;
  const float* y; const int* inv; const float* wts; const int* ids;      // pair p's row of y: inv[p] (inv null: p); ids[p] < 0: none
  const float* shared; const float* sg; const float* self_w; const void* self_x;
  const float* scale;                           // [H] (null: 1)
  const float* post_w;                          // [H]: the update is RMS-normed with this weight (null: it is not)
  // the new rows
  const float* w; const float* b;
  void* out; float* out32;
  int H, slots, norm, one_plus;                 // norm: 0 none, 1 RMS (w or 1 + w), 2 layer norm (w, b)
  float eps, post_eps;
};

}  // namespace spark
