// Row kernels of the parallel block (one norm feeds a mixer and a feed-forward, both outputs are added together), for
// bf16 and fp32 activations.  The residual stream, norms, token-shift state and decays are fp32 in both.
//
//   embed_scaled      x = table[id] * scale
//   add_norm_rows     res += delta;  h = RMSNorm(res) * (w or 1 + w), optionally a second fp32 copy of h
//   token_shift       five mixes h + (h' - h) mu_s of the current and the previous row of the sequence
//   channel_decay     log decay  -exp(W2 tanh(z) + w0)  per channel, fp32 throughout
//   gate_concat       [ group-RMSNorm(o) * w * gate(g) | gelu(gate) * up ]: the input row of the block's single output
//                     product (the mixer's output matrix and the down projection are stored side by side along K)
#include "../common/rows.cuh"

namespace spark {

template <typename TW>
__global__ void __launch_bounds__(128)
embed_scaled_kernel(const TW* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out, int H, int V,
                    float scale, int* __restrict__ status) {
  pdl_wait();
  const int r = blockIdx.x, id = ids[r];
  const bool ok = id >= 0 && id < V;                        // an id outside the table: zero row + status word
  if (!ok && threadIdx.x == 0 && status) set_status(status, ST_BOUNDS, r, id, V);
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    out[static_cast<size_t>(r) * H + i] = ok ? ldf(table + static_cast<size_t>(id) * H + i) * scale : 0.f;
}

template <typename TO>
__global__ void __launch_bounds__(256)
add_norm_rows_kernel(const float* __restrict__ delta, float* __restrict__ res, const float* __restrict__ w,
                     TO* __restrict__ out, float* __restrict__ out32, int H, float eps, int one_plus) {
  __shared__ float sh[32];
  pdl_wait();
  const size_t row = static_cast<size_t>(blockIdx.x) * H;
  float* x = res + row;
  const bool vec = (H & 3) == 0;
  float ss = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      float4 v = ldf4(x + i);
      if (delta != nullptr) {
        const float4 d = ldf4(delta + row + i);
        v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
        stf4(x + i, v);
      }
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float v = x[i];
      if (delta != nullptr) { v += delta[row + i]; x[i] = v; }
      ss += v * v;
    }
  }
  const float rs = 1.f / sqrtf(block_sum_all(ss, sh) / H + eps);
  const float one = one_plus ? 1.f : 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      const float4 v = ldf4(x + i), g = ldf4(w + i);
      const float4 y = make_float4(v.x * rs * (one + g.x), v.y * rs * (one + g.y), v.z * rs * (one + g.z), v.w * rs * (one + g.w));
      if (out != nullptr) stf4(out + row + i, y);
      if (out32 != nullptr) stf4(out32 + row + i, y);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float y = x[i] * rs * (one + w[i]);
      if (out != nullptr) stf(out + row + i, y);
      if (out32 != nullptr) out32[row + i] = y;
    }
  }
}

// grid (R, ceil(H / 1024)); 256 threads x 4 channels.  The first row of a segment reads the carried row of its slot.
template <typename TO>
__global__ void __launch_bounds__(256)
token_shift_kernel(const float* __restrict__ h, const float* __restrict__ carried, const int* __restrict__ row_slot,
                   const int* __restrict__ row_j, const float* __restrict__ mu, int n_mix, TO* __restrict__ out, int R, int H) {
  pdl_wait();
  const int r = blockIdx.x;
  const float* cur = h + static_cast<size_t>(r) * H;
  const float* prev = row_j[r] > 0 ? cur - H : carried + static_cast<size_t>(row_slot[r]) * H;
  const int i0 = blockIdx.y * 1024 + threadIdx.x * 4;
  if ((H & 3) == 0) {
    if (i0 >= H) return;
    const float4 c = ldf4(cur + i0), p = ldf4(prev + i0);
    for (int s = 0; s < n_mix; ++s) {
      const float4 m = ldf4(mu + static_cast<size_t>(s) * H + i0);
      stf4(out + (static_cast<size_t>(s) * R + r) * H + i0,
           make_float4(c.x + (p.x - c.x) * m.x, c.y + (p.y - c.y) * m.y, c.z + (p.z - c.z) * m.z, c.w + (p.w - c.w) * m.w));
    }
  } else {
    for (int i = i0; i < min(i0 + 4, H); ++i)
      for (int s = 0; s < n_mix; ++s)
        stf(out + (static_cast<size_t>(s) * R + r) * H + i, cur[i] + (prev[i] - cur[i]) * mu[static_cast<size_t>(s) * H + i]);
  }
}

// log of the decay exp(-exp(x)), bounded where the decay itself is 0 in fp32 (differences of its running sums stay exact)
__device__ __forceinline__ float log_decay(float x) { return fmaxf(-expf(x), -105.f); }

// grid (ceil(N / 32), ceil(R / RB)); 128 threads: four lanes per channel (eight ranks each in turn), RB rows per CTA.
// rank is a multiple of 8.
template <typename TW, int RB>
__global__ void __launch_bounds__(128)
channel_decay_kernel(const float* __restrict__ z, int ldz, const TW* __restrict__ w2, int ldw, int rank,
                     const float* __restrict__ w0, float* __restrict__ logw, int R, int N) {
  extern __shared__ float t[];                               // [rank][RB]
  const int d = blockIdx.x * 32 + (threadIdx.x >> 2), part = threadIdx.x & 3, r0 = blockIdx.y * RB;
  pdl_wait();
  for (int i = threadIdx.x; i < rank * RB; i += 128) {
    const int k = i / RB, r = r0 + i % RB;
    t[i] = r < R ? tanhf(z[static_cast<size_t>(r) * ldz + k]) : 0.f;
  }
  __syncthreads();
  float acc[RB];
#pragma unroll
  for (int r = 0; r < RB; ++r) acc[r] = 0.f;
  if (d < N)
    for (int k0 = part * 8; k0 < rank; k0 += 32) {
      const TW* wr = w2 + static_cast<size_t>(d) * ldw + k0;
      const float4 a = ldf4(wr), b = ldf4(wr + 4);
      const float w[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int k = 0; k < 8; ++k)
#pragma unroll
        for (int r = 0; r < RB; ++r) acc[r] = fmaf(w[k], t[(k0 + k) * RB + r], acc[r]);
    }
#pragma unroll
  for (int r = 0; r < RB; ++r) {
    float v = acc[r];
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    if (d < N && (r & 3) == part && r0 + r < R) logw[static_cast<size_t>(r0 + r) * N + d] = log_decay(v + w0[d]);
  }
}

// z [R, N] fp32 holds W2 tanh(..) already (prefill: a tensor-core product): z <- -exp(z + w0), in place.
__global__ void __launch_bounds__(256)
neg_exp_bias_kernel(float* __restrict__ z, const float* __restrict__ w0, long long n, int N) {
  for (long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x; i < n; i += static_cast<long long>(gridDim.x) * 256)
    z[i] = log_decay(z[i] + w0[i % N]);
}

// [R, ld] fp32 -> tanh as a two-term bf16 sum: out[r] = [hi (n) | lo (n)], so that one bf16 product against [W | W]
// carries 16 significant bits of the activation.
__global__ void __launch_bounds__(256)
tanh_split_kernel(const float* __restrict__ z, int ldz, __nv_bfloat16* __restrict__ out, int R, int n) {
  for (int i = blockIdx.x * 256 + threadIdx.x; i < R * n; i += gridDim.x * 256) {
    const int r = i / n, k = i - r * n;
    const float v = tanhf(z[static_cast<size_t>(r) * ldz + k]);
    const __nv_bfloat16 hi = __float2bfloat16(v);
    out[static_cast<size_t>(r) * 2 * n + k] = hi;
    out[static_cast<size_t>(r) * 2 * n + n + k] = __float2bfloat16(v - __bfloat162float(hi));
  }
}

// grid (R, 1 + ceil(F / 1024)); 256 threads.  blockIdx.y == 0: the mixer part (columns [0, N), zero up to `off`); the
// other blocks: 1024 feed-forward columns each (columns [off, off + F), the last one zeroes the padding up to ldo).
// group = columns that are normalised together (0: no norm).  gate_kind: 0 none, 1 sigmoid, 2 silu; a gate column per
// output column, or per `gate_div` output columns (one per head).
template <typename T>
__global__ void __launch_bounds__(256)
gate_concat_kernel(const float* __restrict__ o, int ldin, int N, int group, const float* __restrict__ w, float eps,
                   const T* __restrict__ gate, int ldg, int gate_kind, int gate_div, const T* __restrict__ ff, int ldff, int up_off,
                   int F, T* __restrict__ out, int ldo, int off, int vec) {
  // vec: every row start the kernel touches is 4-element aligned and groups are multiples of 4 columns
  __shared__ float sh[32];
  pdl_wait();
  const int r = blockIdx.x;
  T* orow = out + static_cast<size_t>(r) * ldo;
  if (blockIdx.y > 0) {
    const T* fr = ff + static_cast<size_t>(r) * ldff;
    const int base = (blockIdx.y - 1) * 1024;
    const int i4 = base + threadIdx.x * 4;
    if (vec) {                                                // four columns per thread
      if (i4 >= ldo - off) return;
      if (i4 + 4 <= F) {
        const float4 g = ldf4(fr + i4), u = ldf4(fr + up_off + i4);
        stf4(orow + off + i4, make_float4(gelu_tanh_t<T>(g.x) * u.x, gelu_tanh_t<T>(g.y) * u.y, gelu_tanh_t<T>(g.z) * u.z,
                                          gelu_tanh_t<T>(g.w) * u.w));
        return;
      }
      for (int i = i4; i < min(i4 + 4, ldo - off); ++i) stf(orow + off + i, i < F ? gelu_tanh_t<T>(ldf(fr + i)) * ldf(fr + up_off + i) : 0.f);
      return;
    }
    for (int i = base + threadIdx.x; i < min(base + 1024, ldo - off); i += 256)
      stf(orow + off + i, i < F ? gelu_tanh_t<T>(ldf(fr + i)) * ldf(fr + up_off + i) : 0.f);
    return;
  }
  if (o == nullptr) return;
  const float* x = o + static_cast<size_t>(r) * ldin;
  const T* gr = gate ? gate + static_cast<size_t>(r) * ldg : nullptr;
  auto put = [&](int i, float rs) {
    float v = x[i] * rs;
    if (w) v *= w[i];
    if (gate_kind == 1) v *= sigmoid_t<T>(ldf(gr + i / gate_div));
    else if (gate_kind == 2) v *= silu_t<T>(ldf(gr + i / gate_div));
    stf(orow + i, v);
  };
  if (vec && group > 0 && gate_kind > 0 && w != nullptr) {
    auto put4 = [&](int i, float4 v, float rs) {
      const float4 ww = ldf4(w + i), g = ldf4(gr + i);
      const bool sg = gate_kind == 1;
      v.x *= rs * ww.x * (sg ? sigmoid_t<T>(g.x) : silu_t<T>(g.x)); v.y *= rs * ww.y * (sg ? sigmoid_t<T>(g.y) : silu_t<T>(g.y));
      v.z *= rs * ww.z * (sg ? sigmoid_t<T>(g.z) : silu_t<T>(g.z)); v.w *= rs * ww.w * (sg ? sigmoid_t<T>(g.w) : silu_t<T>(g.w));
      stf4(orow + i, v);
    };
    if (group == N) {
      float ss = 0.f;
      for (int i = threadIdx.x * 4; i < N; i += 1024) { const float4 v = ldf4(x + i); ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
      const float rs = 1.f / sqrtf(block_sum_all(ss, sh) / N + eps);
      for (int i = threadIdx.x * 4; i < N; i += 1024) put4(i, ldf4(x + i), rs);
    } else {
      const int lane = threadIdx.x & 31;
      for (int g = threadIdx.x >> 5; g < N / group; g += 8) {
        float ss = 0.f;
        for (int i = lane * 4; i < group; i += 128) { const float4 v = ldf4(x + g * group + i); ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
        const float rs = 1.f / sqrtf(warp_sum(ss) / group + eps);
        for (int i = lane * 4; i < group; i += 128) put4(g * group + i, ldf4(x + g * group + i), rs);
      }
    }
    for (int i = N + threadIdx.x; i < off; i += 256) stf(orow + i, 0.f);
    return;
  }
  if (group == N && group > 0) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < N; i += 256) ss = fmaf(x[i], x[i], ss);
    const float rs = 1.f / sqrtf(block_sum_all(ss, sh) / N + eps);
    for (int i = threadIdx.x; i < N; i += 256) put(i, rs);
  } else if (group > 0) {                                     // a warp per group
    const int lane = threadIdx.x & 31;
    for (int g = threadIdx.x >> 5; g < N / group; g += 8) {
      float ss = 0.f;
      for (int i = lane; i < group; i += 32) ss = fmaf(x[g * group + i], x[g * group + i], ss);
      const float rs = 1.f / sqrtf(warp_sum(ss) / group + eps);
      for (int i = lane; i < group; i += 32) put(g * group + i, rs);
    }
  } else {
    for (int i = threadIdx.x; i < N; i += 256) put(i, 1.f);
  }
  for (int i = N + threadIdx.x; i < off; i += 256) stf(orow + i, 0.f);
}

}  // namespace spark

using namespace spark;

#define SPARK_BY_TYPE(f32, CALL)          \
  if (f32) { using T = float; CALL; }     \
  else { using T = __nv_bfloat16; CALL; }

extern "C" int spark_embed_scaled(const void* table, const int* ids, float* out, int R, int H, int V, float scale, int f32,
                                  int* status, cudaStream_t s) {
  if (R <= 0) return 0;
  SPARK_BY_TYPE(f32, spark_launch_pdl(embed_scaled_kernel<T>, dim3(R), dim3(128), 0, s, dim3(1, 1, 1), (const T*)table, ids, out,
                                      H, V, scale, status))
  return spark_launch_rc(__func__);
}

extern "C" int spark_add_norm_rows(const float* delta, float* res, const float* w, void* out, float* out32, int R, int H,
                                   float eps, int one_plus, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  SPARK_BY_TYPE(f32, spark_launch_pdl(add_norm_rows_kernel<T>, dim3(R), dim3(256), 0, s, dim3(1, 1, 1), delta, res, w, (T*)out,
                                      out32, H, eps, one_plus))
  return spark_launch_rc(__func__);
}

extern "C" int spark_token_shift(const float* h, const float* carried, const int* row_slot, const int* row_j, const float* mu,
                                 int n_mix, void* out, int R, int H, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  SPARK_BY_TYPE(f32, spark_launch_pdl(token_shift_kernel<T>, dim3(R, (H + 1023) / 1024), dim3(256), 0, s, dim3(1, 1, 1), h, carried,
                                      row_slot, row_j, mu, n_mix, (T*)out, R, H))
  return spark_launch_rc(__func__);
}

extern "C" int spark_channel_decay(const float* z, int ldz, const void* w2, int ldw, int rank, const float* w0, float* logw,
                                   int R, int N, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  if (rank <= 0 || (rank & 7) || (ldw & 7) || rank * 64 > 48 * 1024) return -5;
#define SPARK_CHD(RB)                                                                                                     \
  spark_launch_pdl(channel_decay_kernel<T, RB>, dim3((N + 31) / 32, (R + RB - 1) / RB), dim3(128), rank * RB * 4, s,      \
                   dim3(1, 1, 1), z, ldz, (const T*)w2, ldw, rank, w0, logw, R, N)
  SPARK_BY_TYPE(f32, if (R <= 4) SPARK_CHD(4); else SPARK_CHD(16))
#undef SPARK_CHD
  return spark_launch_rc(__func__);
}

extern "C" int spark_neg_exp_bias(float* z, const float* w0, int R, int N, cudaStream_t s) {
  if (R <= 0) return 0;
  const long long n = static_cast<long long>(R) * N;
  neg_exp_bias_kernel<<<static_cast<int>(n / 1024 + 1 < 1184 ? n / 1024 + 1 : 1184), 256, 0, s>>>(z, w0, n, N);
  return spark_launch_rc(__func__);
}

extern "C" int spark_tanh_split(const float* z, int ldz, void* out, int R, int n, cudaStream_t s) {
  if (R <= 0) return 0;
  tanh_split_kernel<<<R * n / 512 + 1, 256, 0, s>>>(z, ldz, (__nv_bfloat16*)out, R, n);
  return spark_launch_rc(__func__);
}

extern "C" int spark_gate_concat(const float* o, int ldin, int N, int group, const float* w, float eps, const void* gate, int ldg,
                                 int gate_kind, int gate_div, const void* ff, int ldff, int up_off, int F, void* out, int ldo,
                                 int off, int R, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  if (group > 0 && N % group) return -5;
  const int nff = ff ? (ldo - off + 1023) / 1024 : 0;
  const uintptr_t a16 = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(w);
  const uintptr_t a8 = reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(ff) | reinterpret_cast<uintptr_t>(out);
  const int vec = ((a16 | (f32 ? a8 : 0)) & 15) == 0 && (a8 & 7) == 0 && gate_div == 1 &&
                  ((ldin | N | group | (gate ? ldg : 0) | (ff ? ldff | up_off : 0) | ldo | off) & 3) == 0;
  SPARK_BY_TYPE(f32, spark_launch_pdl(gate_concat_kernel<T>, dim3(R, 1 + nff), dim3(256), 0, s, dim3(1, 1, 1), o, ldin, N, group, w,
                                      eps, (const T*)gate, ldg, gate_kind, gate_div, (const T*)ff, ldff, up_off, F, (T*)out, ldo, off,
                                      vec))
  return spark_launch_rc(__func__);
}
