// Row kernels of the models whose layers carry their own sizes, for bf16 and fp32 activations.  The residual stream, norms,
// token-shift state and decays are fp32 in both.
//
//   embed_scaled      x = table[id] * scale (+ the sines and cosines of the position)
//   row_update        res += an update (plain rows or the slots of a routed feed-forward; per-channel scale, or RMS-normed);
//                     h = norm of the new residual (RMS, layer norm, or the residual itself), optionally an fp32 copy of h
//   token_shift       five mixes h + (h' - h) mu_s of the current and the previous row of the sequence
//   channel_decay     log decay  -exp(W2 tanh(z) + w0)  or  ln(sigmoid(W2 z + w0)) / tau  per channel, fp32 throughout
//   swiglu_rows       gated activation (out_act.cuh) of [gate | up] rows, both times a weight per row if given
//   gate_concat       [ group-RMSNorm(o) * w * gate(g) | gelu(gate) * up ]: the input row of the block's single output
//                     product (the mixer's output matrix and the down projection are stored side by side along K)
#include "../common/row_update.cuh"
#include "../common/out_act.cuh"

namespace spark {

// pos (optional): channel 2i gets the sine of pos * freq[i], channel 2i + 1 its cosine on top.
template <typename TW>
__global__ void __launch_bounds__(128)
embed_scaled_kernel(const TW* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out, int H, int V,
                    float scale, const int* __restrict__ pos, const double* __restrict__ freq, int* __restrict__ status) {
  pdl_wait();
  const int r = blockIdx.x, id = ids[r];
  const bool ok = id >= 0 && id < V;                        // an id outside the table: zero row + status word
  if (!ok && threadIdx.x == 0 && status) set_status(status, ST_BOUNDS, r, id, V);
  const TW* row = table + static_cast<size_t>(ok ? id : 0) * H;
  float* o = out + static_cast<size_t>(r) * H;
  if (pos == nullptr) {
    for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = ok ? ldf(row + i) * scale : 0.f;
    return;
  }
  const double p = pos[r];
  for (int i = threadIdx.x * 2; i < H; i += blockDim.x * 2) {
    float sn, cs;
    sincosf(static_cast<float>(p * freq[i >> 1]), &sn, &cs);
    o[i] = ok ? ldf(row + i) * scale + sn : 0.f;
    if (i + 1 < H) o[i + 1] = ok ? ldf(row + i + 1) * scale + cs : 0.f;
  }
}

// One CTA per row.  NV > 0: every thread keeps NV groups of four channels in registers (blockDim * 4 * NV >= H, H % 4 == 0,
// 16-byte aligned rows); NV == 0: any width, values are read again.
template <typename T, int NV>
__global__ void __launch_bounds__(NV <= 2 ? 1024 : 256)
row_update_kernel(const __grid_constant__ RowUpdate a) {
  __shared__ float sh[32];
  pdl_wait();
  const int r = blockIdx.x, H = a.H, t = threadIdx.x, nt = blockDim.x;
  const size_t row = static_cast<size_t>(r) * H;
  float* x = a.res + row;
  const bool has = a.delta != nullptr || a.y != nullptr;
  const float sg = a.shared ? (a.sg ? a.sg[r] : 1.f) : 0.f, own = a.self_w ? a.self_w[r] : 0.f;
  const T* sx = static_cast<const T*>(a.self_x) + (a.self_w ? row : 0);
  T* out = static_cast<T*>(a.out) + row;
  const float one = a.one_plus ? 1.f : 0.f;
  if constexpr (NV > 0) {
    float4 v[NV], u[NV];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (t + k * nt) * 4;
      u[k] = v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i >= H) continue;
      v[k] = ldf4(x + i);
      if (a.delta) u[k] = ldf4(a.delta + row + i);
      else if (a.y) {
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s0 = 0; s0 < a.slots; s0 += 4) {           // four slots' rows in flight, added in slot order
          float4 p[4]; float w[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int pi = r * a.slots + s0 + q;
            const bool live = s0 + q < a.slots && a.ids[pi] >= 0;
            w[q] = live ? (a.wts ? a.wts[pi] : 1.f) : 0.f;
            p[q] = live ? __ldcg(reinterpret_cast<const float4*>(a.y + static_cast<size_t>(a.inv ? a.inv[pi] : pi) * H + i))
                        : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            s.x = fmaf(w[q], p[q].x, s.x); s.y = fmaf(w[q], p[q].y, s.y); s.z = fmaf(w[q], p[q].z, s.z); s.w = fmaf(w[q], p[q].w, s.w);
          }
        }
        if (own != 0.f) {
          const float4 p = ldf4(sx + i);
          s.x = fmaf(own, p.x, s.x); s.y = fmaf(own, p.y, s.y); s.z = fmaf(own, p.z, s.z); s.w = fmaf(own, p.w, s.w);
        }
        if (a.shared) {
          const float4 p = ldf4(a.shared + row + i);
          s.x = fmaf(sg, p.x, s.x); s.y = fmaf(sg, p.y, s.y); s.z = fmaf(sg, p.z, s.z); s.w = fmaf(sg, p.w, s.w);
        }
        u[k] = s;
      }
      ss += u[k].x * u[k].x + u[k].y * u[k].y + u[k].z * u[k].z + u[k].w * u[k].w;
    }
    const float ps = a.post_w ? 1.f / sqrtf(block_sum_all(ss, sh) / H + a.post_eps) : 1.f;
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (t + k * nt) * 4;
      if (i >= H) continue;
      if (has) {
        float4 m = make_float4(1.f, 1.f, 1.f, 1.f);
        if (a.scale) m = ldf4(a.scale + i);
        if (a.post_w) { const float4 p = ldf4(a.post_w + i); m.x *= ps * p.x; m.y *= ps * p.y; m.z *= ps * p.z; m.w *= ps * p.w; }
        v[k].x += u[k].x * m.x; v[k].y += u[k].y * m.y; v[k].z += u[k].z * m.z; v[k].w += u[k].w * m.w;
        stf4(x + i, v[k]);
      }
      sum += a.norm == 2 ? v[k].x + v[k].y + v[k].z + v[k].w : v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
    float mean = 0.f, rs = 1.f;
    if (a.norm) {
      sum = block_sum_all(sum, sh) / H;
      if (a.norm == 2) {
        mean = sum;
        float q = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
          if ((t + k * nt) * 4 >= H) continue;
          const float dx = v[k].x - mean, dy = v[k].y - mean, dz = v[k].z - mean, dw = v[k].w - mean;
          q += dx * dx + dy * dy + dz * dz + dw * dw;
        }
        sum = block_sum_all(q, sh) / H;
      }
      rs = 1.f / sqrtf(sum + a.eps);
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (t + k * nt) * 4;
      if (i >= H) continue;
      float4 y = v[k];
      if (a.norm) {
        const float4 g = ldf4(a.w + i);
        y = make_float4((y.x - mean) * rs * (one + g.x), (y.y - mean) * rs * (one + g.y), (y.z - mean) * rs * (one + g.z),
                        (y.w - mean) * rs * (one + g.w));
        if (a.norm == 2) { const float4 b = ldf4(a.b + i); y.x += b.x; y.y += b.y; y.z += b.z; y.w += b.w; }
      }
      if (a.out) stf4(out + i, y);
      if (a.out32) stf4(a.out32 + row + i, y);
    }
  } else {
    auto update = [&](int i) {
      if (a.delta) return a.delta[row + i];
      float s = 0.f;
      for (int k = 0; k < a.slots; ++k) {
        const int pi = r * a.slots + k;
        if (a.ids[pi] >= 0) s = fmaf(a.wts ? a.wts[pi] : 1.f, a.y[static_cast<size_t>(a.inv ? a.inv[pi] : pi) * H + i], s);
      }
      if (own != 0.f) s = fmaf(own, ldf(sx + i), s);
      if (a.shared) s = fmaf(sg, a.shared[row + i], s);
      return s;
    };
    float ps = 1.f;
    if (has && a.post_w) {
      float ss = 0.f;
      for (int i = t; i < H; i += nt) { const float u = update(i); ss = fmaf(u, u, ss); }
      ps = 1.f / sqrtf(block_sum_all(ss, sh) / H + a.post_eps);
    }
    float sum = 0.f;
    for (int i = t; i < H; i += nt) {
      float v = x[i];
      if (has) {
        v += update(i) * (a.scale ? a.scale[i] : 1.f) * (a.post_w ? ps * a.post_w[i] : 1.f);
        x[i] = v;
      }
      sum += a.norm == 2 ? v : v * v;
    }
    float mean = 0.f, rs = 1.f;
    if (a.norm) {
      sum = block_sum_all(sum, sh) / H;
      if (a.norm == 2) {
        mean = sum;
        float q = 0.f;
        for (int i = t; i < H; i += nt) { const float d = x[i] - mean; q = fmaf(d, d, q); }
        sum = block_sum_all(q, sh) / H;
      }
      rs = 1.f / sqrtf(sum + a.eps);
    }
    for (int i = t; i < H; i += nt) {
      float y = x[i];
      if (a.norm) y = (y - mean) * rs * (one + a.w[i]) + (a.norm == 2 ? a.b[i] : 0.f);
      if (a.out) stf(out + i, y);
      if (a.out32) a.out32[row + i] = y;
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
// rank is a multiple of 8.  inv_tau 0: -exp(W2 tanh(z) + w0); else ln(sigmoid(W2 z + w0)) * inv_tau.
template <typename TZ, typename TW, int RB>
__global__ void __launch_bounds__(128)
channel_decay_kernel(const TZ* __restrict__ z, int ldz, const TW* __restrict__ w2, int ldw, int rank,
                     const float* __restrict__ w0, float* __restrict__ logw, int R, int N, float inv_tau) {
  extern __shared__ float t[];                               // [rank][RB]
  const int d = blockIdx.x * 32 + (threadIdx.x >> 2), part = threadIdx.x & 3, r0 = blockIdx.y * RB;
  pdl_wait();
  for (int i = threadIdx.x; i < rank * RB; i += 128) {
    const int k = i / RB, r = r0 + i % RB;
    const float x = r < R ? ldf(z + static_cast<size_t>(r) * ldz + k) : 0.f;
    t[i] = inv_tau > 0.f ? x : tanhf(x);
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
    if (d < N && (r & 3) == part && r0 + r < R) logw[static_cast<size_t>(r0 + r) * N + d] = inv_tau > 0.f ? log_sigmoid_decay(v + w0[d], inv_tau) : log_decay(v + w0[d]);
  }
}

// The log-sigmoid form for many rows: a channel per thread, 32 rows per CTA.  grid (ceil(N / 128), ceil(R / 32)); 128 threads.
template <typename T>
__global__ void __launch_bounds__(128)
log_sigmoid_decay_rows_kernel(const T* __restrict__ z, int ldz, const T* __restrict__ w2, int ldw, int rank, const float* __restrict__ b,
                              float inv_tau, float* __restrict__ logw, int R, int N) {
  constexpr int RB = 32;
  extern __shared__ __align__(16) float t[];                 // [rank][RB]
  const int d = blockIdx.x * 128 + threadIdx.x, r0 = blockIdx.y * RB;
  pdl_wait();
  for (int i = threadIdx.x; i < rank * RB; i += 128) {
    const int r = i / rank, k = i - r * rank;
    t[k * RB + r] = r0 + r < R ? ldf(z + static_cast<size_t>(r0 + r) * ldz + k) : 0.f;
  }
  __syncthreads();
  if (d >= N) return;
  float acc[RB];
#pragma unroll
  for (int r = 0; r < RB; ++r) acc[r] = 0.f;
  for (int k0 = 0; k0 < rank; k0 += 8) {
    const T* wr = w2 + static_cast<size_t>(d) * ldw + k0;
    const float4 p = ldf4(wr), q = ldf4(wr + 4);
    const float w[8] = {p.x, p.y, p.z, p.w, q.x, q.y, q.z, q.w};
#pragma unroll
    for (int k = 0; k < 8; ++k)
#pragma unroll
      for (int r = 0; r < RB; r += 4) {
        const float4 x = *reinterpret_cast<const float4*>(t + (k0 + k) * RB + r);
        acc[r] = fmaf(w[k], x.x, acc[r]); acc[r + 1] = fmaf(w[k], x.y, acc[r + 1]);
        acc[r + 2] = fmaf(w[k], x.z, acc[r + 2]); acc[r + 3] = fmaf(w[k], x.w, acc[r + 3]);
      }
  }
  const float bias = b[d];
#pragma unroll
  for (int r = 0; r < RB; ++r)
    if (r0 + r < R) logw[static_cast<size_t>(r0 + r) * N + d] = log_sigmoid_decay(acc[r] + bias, inv_tau);
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

// grid (ceil(F / 1024), rows); 256 threads x 4 columns of [gate (F) | up (F)].  wts (optional): the weight of row r's pair is
// wts[perm ? perm[r] : r].
template <typename T>
__global__ void __launch_bounds__(256)
swiglu_rows_kernel(const T* __restrict__ gu, int ldi, int F, const float* __restrict__ wts, const int* __restrict__ perm,
                   T* __restrict__ out, int ldo, int R, GluAct act) {
  pdl_wait();
  const int i = blockIdx.x * 1024 + threadIdx.x * 4;
  if (i >= F) return;
  for (int r = blockIdx.y; r < R; r += gridDim.y) {
    const T* x = gu + static_cast<size_t>(r) * ldi + i;
    const float4 g = ldf4(x), u = ldf4(x + F);
    const float w = wts ? wts[perm ? perm[r] : r] : 1.f;
    stf4(out + static_cast<size_t>(r) * ldo + i, make_float4(glu_t<T>(act, w * g.x, w * u.x), glu_t<T>(act, w * g.y, w * u.y),
                                                             glu_t<T>(act, w * g.z, w * u.z), glu_t<T>(act, w * g.w, w * u.w)));
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

extern "C" int spark_embed_scaled(const void* table, const int* ids, float* out, int R, int H, int V, float scale, const int* pos,
                                  const double* freq, int f32, int* status, cudaStream_t s) {
  if (R <= 0) return 0;
  if (pos && !freq) return -5;
  SPARK_BY_TYPE(f32, spark_launch_pdl(embed_scaled_kernel<T>, dim3(R), dim3(128), 0, s, dim3(1, 1, 1), (const T*)table, ids, out,
                                      H, V, scale, pos, freq, status))
  return spark_launch_rc(__func__);
}

extern "C" int spark_row_update(const RowUpdate* u, int R, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  if (u->y && (u->slots <= 0 || !u->ids)) return -5;
  if ((u->norm && !u->w) || (u->norm == 2 && !u->b) || (u->self_w && !u->self_x)) return -5;
  const uintptr_t al = reinterpret_cast<uintptr_t>(u->res) | reinterpret_cast<uintptr_t>(u->delta) | reinterpret_cast<uintptr_t>(u->y) |
                       reinterpret_cast<uintptr_t>(u->shared) | reinterpret_cast<uintptr_t>(u->self_x) | reinterpret_cast<uintptr_t>(u->scale) |
                       reinterpret_cast<uintptr_t>(u->post_w) | reinterpret_cast<uintptr_t>(u->w) | reinterpret_cast<uintptr_t>(u->b) |
                       reinterpret_cast<uintptr_t>(u->out) | reinterpret_cast<uintptr_t>(u->out32);
  const int groups = u->H / 4, warps = (groups + 31) / 32 * 32;
  int th = warps < 256 ? warps : 256;                       // many rows: 256 threads each; few rows: up to 1024
  if (R < 148 && groups <= 2048) th = warps < 1024 ? warps : 1024;
  const int nv = th > 0 ? (groups + th - 1) / th : 0;
#define SPARK_ROWUP(NV) SPARK_BY_TYPE(f32, spark_launch_pdl(row_update_kernel<T, NV>, dim3(R), dim3(NV ? th : (u->H >= 4096 ? 1024 : 256)), 0, s, dim3(1, 1, 1), *u))
  if ((u->H & 3) || (al & 15) || nv > 8) { SPARK_ROWUP(0) }
  else if (nv <= 1) { SPARK_ROWUP(1) }
  else if (nv <= 2) { SPARK_ROWUP(2) }
  else if (nv <= 4) { SPARK_ROWUP(4) }
  else { SPARK_ROWUP(8) }
#undef SPARK_ROWUP
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
#define SPARK_CHD(TZ, RB, inv_tau)                                                                                        \
  spark_launch_pdl(channel_decay_kernel<TZ, T, RB>, dim3((N + 31) / 32, (R + RB - 1) / RB), dim3(128), rank * RB * 4, s,  \
                   dim3(1, 1, 1), (const TZ*)z, ldz, (const T*)w2, ldw, rank, w0, logw, R, N, inv_tau)
  SPARK_BY_TYPE(f32, if (R <= 4) SPARK_CHD(float, 4, 0.f); else SPARK_CHD(float, 16, 0.f))
  return spark_launch_rc(__func__);
}

// z in the activation type, columns up to the padded rank readable and zero (or w2's columns there zero); tau > 0.
extern "C" int spark_log_sigmoid_decay(const void* z, int ldz, const void* w2, int ldw, int rank, const float* b, float tau, float* logw,
                                       int R, int N, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  if (rank <= 0 || (rank & 7) || (ldw & 7) || rank * 64 > 48 * 1024 || !(tau > 0.f)) return -5;
  const float* w0 = b;
  const float inv_tau = 1.f / tau;
  if (R >= 64 && rank * 128 <= 48 * 1024) {
    SPARK_BY_TYPE(f32, spark_launch_pdl(log_sigmoid_decay_rows_kernel<T>, dim3((N + 127) / 128, (R + 31) / 32), dim3(128), rank * 128, s,
                                        dim3(1, 1, 1), (const T*)z, ldz, (const T*)w2, ldw, rank, b, inv_tau, logw, R, N))
    return spark_launch_rc(__func__);
  }
  SPARK_BY_TYPE(f32, if (R <= 4) SPARK_CHD(T, 4, inv_tau); else SPARK_CHD(T, 16, inv_tau))
#undef SPARK_CHD
  return spark_launch_rc(__func__);
}

extern "C" int spark_swiglu_rows(const void* gu, int ldi, int F, const float* wts, const int* perm, void* out, int ldo, int R,
                                 const GluAct* act, int f32, cudaStream_t s) {
  if (R <= 0) return 0;
  if ((F | ldi | ldo) & 7) return -5;
  const dim3 grid((F + 1023) / 1024, R < 65535 ? R : 65535);
  SPARK_BY_TYPE(f32, spark_launch_pdl(swiglu_rows_kernel<T>, grid, dim3(256), 0, s, dim3(1, 1, 1), (const T*)gu, ldi, F, wts, perm, (T*)out,
                                      ldo, R, act ? *act : GluAct{0.f, 1.f, 0.f}))
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
