// Merge of split attention partials: part_o fp32 [R, H, nsplit, L] (unnormalised outputs), part_ml fp32 [R, H, nsplit, 2]
// (maximum, sum); an empty split has maximum -inf and its part_o rows are not read.
#pragma once
#include "decode.cuh"

namespace spark {

// grid (R, ceil(H / hpc)); 256 threads.  Splits merged in ascending order; `sink` (per head, optional) joins the
// denominator.  A CTA owns `hpc` heads of one row: the per-head weights of the splits are computed once into shared
// memory, then the threads sweep the hpc x L outputs with 16-byte loads.  The launcher picks hpc so that a decode
// round of a few rows still fills the SMs (one head per CTA), while a prefill chunk keeps one CTA per row.
static __global__ void __launch_bounds__(256)
split_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int nsplit, const float* __restrict__ sink,
                   int H, int L, int hpc, __nv_bfloat16* __restrict__ out, const __nv_bfloat16* __restrict__ gate, int ldg,
                   const int* __restrict__ rows, int out_by_row, int ldo, float out_scale) {
  // out_by_row: result of launch row r goes to row rows[r] of `out` instead of row r
  // gate (optional): one logit per head in the row's gate columns, the head's output is scaled by its sigmoid; out_scale: a
  // constant factor; ldo: row stride of `out` (heads of L columns)
  // The statistics of a head's splits are reduced by one warp (split s in lane s % 32, so empty trailing splits do not
  // change a bit of the result).
  extern __shared__ float wts[];                        // [hpc][nsplit]: exp(m_s - M) / l
  __shared__ int live_s;                                // splits that hold visible tokens
  if (threadIdx.x == 0) live_s = 0;
  __syncthreads();
  const int r = blockIdx.x, h0 = blockIdx.y * hpc;
  const int nh = min(hpc, H - h0);
  const int lane = threadIdx.x & 31;
  for (int hl = threadIdx.x >> 5; hl < nh; hl += blockDim.x >> 5) {
    const int h = h0 + hl;
    const float2* ml = reinterpret_cast<const float2*>(part_ml) + (static_cast<size_t>(r) * H + h) * nsplit;
    float M = sink ? sink[h] : -INFINITY;
    int live = 0;
    for (int s = lane; s < nsplit; s += 32) {
      const float m = ml[s].x;
      M = fmaxf(M, m);
      if (m != -INFINITY) live = s + 1;
    }
    M = warp_max(M);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) live = max(live, __shfl_xor_sync(0xffffffffu, live, o));
    float l = 0.f;
    for (int s = lane; s < live; s += 32) {
      const float2 v = ml[s];
      if (v.x != -INFINITY) l += __expf(v.x - M) * v.y;
    }
    l = warp_sum(l) + (sink ? __expf(sink[h] - M) : 0.f);
    float inv = out_scale / l;
    if (gate) inv /= 1.f + expf(-__bfloat162float(gate[static_cast<size_t>(rows ? rows[r] : r) * ldg + h]));
    for (int s = lane; s < live; s += 32) {
      const float m = ml[s].x;
      wts[hl * nsplit + s] = m != -INFINITY ? __expf(m - M) * inv : 0.f;
    }
    for (int s = live + lane; s < nsplit; s += 32) wts[hl * nsplit + s] = 0.f;
    if (lane == 0) atomicMax(&live_s, live);
  }
  __syncthreads();
  const int L4 = L >> 2;
  for (int i = threadIdx.x; i < nh * L4; i += blockDim.x) {
    const int hl = i / L4, d = (i - hl * L4) * 4, h = h0 + hl;
    const size_t pb = (static_cast<size_t>(r) * H + h) * nsplit;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    const int ns = live_s;
    for (int s0 = 0; s0 < ns; s0 += 8) {                 // eight partial rows in flight
      float4 pv[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) pv[u] = __ldcg(reinterpret_cast<const float4*>(part_o + (pb + min(s0 + u, ns - 1)) * L + d));
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const float w = s0 + u < ns ? wts[hl * nsplit + s0 + u] : 0.f;
        const float4 p = pv[u];
        if (w == 0.f) continue;                         // (an empty split's partial rows are not initialised)
        o.x = fmaf(w, p.x, o.x); o.y = fmaf(w, p.y, o.y); o.z = fmaf(w, p.z, o.z); o.w = fmaf(w, p.w, o.w);
      }
    }
    const __nv_bfloat162 b0 = __floats2bfloat162_rn(o.x, o.y), b1 = __floats2bfloat162_rn(o.z, o.w);
    uint2 ov; ov.x = *reinterpret_cast<const uint32_t*>(&b0); ov.y = *reinterpret_cast<const uint32_t*>(&b1);
    *reinterpret_cast<uint2*>(out + static_cast<size_t>(out_by_row && rows ? rows[r] : r) * ldo + h * L + d) = ov;
  }
}

// hpc: heads per CTA -- enough CTAs for two per SM when rows are few.
static inline int launch_split_merge(const float* part_o, const float* part_ml, int nsplit, const float* sink, int R, int H, int L,
                                     void* out, const void* gate, int ldg, const int* rows, int out_by_row, cudaStream_t s, int ldo = 0,
                                     float out_scale = 1.f) {
  int hpc = H;
  while (hpc > 1 && (R * ((H + hpc - 1) / hpc) < 296 || hpc * nsplit * 4 > 48 * 1024)) hpc = (hpc + 1) / 2;
  if (hpc * nsplit * 4 > 48 * 1024) return -6;
  const int L4 = L >> 2;
  const int threads = hpc * L4 >= 256 ? 256 : ((hpc * L4 + 31) / 32 * 32);   // whole warps
  split_merge_kernel<<<dim3(R, (H + hpc - 1) / hpc), threads, hpc * nsplit * 4, s>>>(part_o, part_ml, nsplit, sink, H, L, hpc,
                                                                                  (__nv_bfloat16*)out, (const __nv_bfloat16*)gate, ldg,
                                                                                  rows, out_by_row, ldo ? ldo : H * L, out_scale);
  return 0;
}

}  // namespace spark
