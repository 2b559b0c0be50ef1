// Grouped-query softmax attention over a paged cache (64-token pages of per-token key / value rows), for bf16 and fp32
// activations:
//
//   conv_prep     short causal convolution over time on the stacked [q | k | v] projections: queries to a buffer, keys and
//                 values to their pages; the last taps - 1 projected rows of a sequence are its state
//   head_prep     RMS norm per query / key head, rotation, temperature of the queries; keys and values to their pages (or
//                 queries alone, for a layer that reads another layer's cache)
//   paged_prefill prompts: flash-style tiles on tensor cores, one page of keys per step
//   paged_decode  decode / verify rows: split-KV, a page per split, the query heads of a key / value head as MMA rows
//   paged_rows    one CTA per (row, head) on the FP32 units: the 32-bit mode, and head sizes the others do not cover
//
// Scores are soft-capped (cap * tanh(q.k scale / cap); cap 0: not), get a bias per head and distance (the last entry serves
// everything farther; null: none) or lose slope * distance, and are visible inside the row's aligned chunk of the sequence or a
// window that ends at the row (both 0: everything before it).  An optional sink per head enters the denominator only, an
// optional sigmoid gate per head and a constant scale the outputs.  Scores, softmax and its weights are fp32; the weights enter
// the tensor-core product as two-term bf16 sums.  Head widths are padded to 16.
#include "../common/rows.cuh"
#include "../common/split_merge.cuh"

namespace spark {

constexpr int PGA_PAGE = 64;
constexpr float PGA_LOG2E = 1.4426950408889634f;

struct PagedAttn {
  const void *q, *k, *v;                 // q [rows, ldq]; caches [pages, 64, G * D] / [pages, 64, G * V]
  void* out;                             // [rows, ldo]: heads of V columns
  const int *pos, *rows, *row_slot;      // per plan row; rows: launch row -> plan row (null: identity)
  const int* pages;                      // [slots, page_ld]
  const float *bias, *sink;              // [H, bias_n] / [H]
  float *part_o, *part_ml;
  const int* segs;                       // prompts: slot, first row, rows, first position (stride seg_ld)
  const float* slopes;                   // [H]: taken off per token of distance
  const void* gate;                      // [rows, ldg]: one logit per head
  int page_ld, H, G, D, V, ldq, bias_n, chunk, seg_ld, nsplit, window, ldg, ldo;
  float scale, cap, out_scale;
};

__device__ __forceinline__ int first_visible(int p, const PagedAttn& a) {
  return a.chunk > 0 ? p / a.chunk * a.chunk : (a.window > 0 ? max(p - a.window + 1, 0) : 0);
}
// factor of head h's output in plan row pr
template <typename T>
__device__ __forceinline__ float head_factor(const PagedAttn& a, int pr, int h) {
  return a.gate ? a.out_scale * sigmoid_f(ldf(static_cast<const T*>(a.gate) + static_cast<size_t>(pr) * a.ldg + h)) : a.out_scale;
}

// tanh to fp32 accuracy in the sense of the soft cap: the Taylor polynomial near 0 (where the quotient form would cancel),
// 1 - 2 / (exp(2z) + 1) elsewhere (absolute error of a few 2^-23).  The polynomial gives tanh(z) / z.
constexpr float CAP_NEAR = 0.25f;
__device__ __forceinline__ float tanh_over_z(float z) {
  const float s = z * z;
  return fmaf(s, fmaf(s, fmaf(s, fmaf(s, 62.f / 2835.f, -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), 1.f);
}
__device__ __forceinline__ float cap_tanh(float z) {
  const float near = z * tanh_over_z(z), far = 1.f - __fdividef(2.f, 1.f + __expf(2.f * fminf(z, 40.f)));
  return fabsf(z) < CAP_NEAR ? near : far;
}

// ------------------------------------------------------------------------------------------------ short convolution
struct ConvPrep {
  const void* proj; const float* w;      // [rows, ldp]; [taps, C]
  void *tail, *q, *k, *v;                // tail [slots, taps - 1, C]
  const int *segs, *n_rows, *pages;      // n_rows (optional): rows of a segment that the tail advances by
  int* status;
  int ldp, C, taps, nq, nk, nv, page_ld, tile, commit, store;
};

// grid (row tiles, channel blocks, segments); 128 threads x 16 bytes of channels.  TAPS > 0: the window lives in registers.
// Only the first tile of a segment reads the tail (tile >= taps - 1), and the same thread advances it afterwards.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
conv_prep_kernel(const __grid_constant__ ConvPrep a) {
  constexpr int VEC = 16 / sizeof(T), NV4 = VEC / 4;
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : a.taps, past = taps - 1;
  const int c0 = (blockIdx.y * 128 + threadIdx.x) * VEC;
  const int* sg = a.segs + blockIdx.z * 4;
  const int slot = sg[0], r0 = sg[1], n = sg[2], pos0 = sg[3], j0 = blockIdx.x * a.tile;
  if (c0 >= a.C || j0 >= n) return;
  const T* proj = static_cast<const T*>(a.proj) + static_cast<size_t>(r0) * a.ldp + c0;
  T* tail = static_cast<T*>(a.tail) + static_cast<size_t>(slot) * past * a.C + c0;
  auto load = [&](int j, float (&u)[VEC]) {                  // projected row j of the segment; j < 0: the sequence's past
    const T* p = j >= 0 ? proj + static_cast<size_t>(j) * a.ldp : tail + static_cast<size_t>(past + j) * a.C;
#pragma unroll
    for (int i = 0; i < NV4; ++i) {
      const float4 f = ldf4(p + 4 * i);
      u[4 * i] = f.x; u[4 * i + 1] = f.y; u[4 * i + 2] = f.z; u[4 * i + 3] = f.w;
    }
  };
  if (a.store) {
    constexpr int WIN = TAPS > 1 ? TAPS - 1 : 1;
    float win[WIN][VEC], w[TAPS > 0 ? TAPS : 1][VEC];
    if (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < TAPS; ++i)
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[i][e] = a.w[static_cast<size_t>(i) * a.C + c0 + e];
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i) load(j0 - past + i, win[i]);
    }
    const int jn = min(n, j0 + a.tile);
    for (int j = j0; j < jn; ++j) {
      float y[VEC], u[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = 0.f;
      if (TAPS > 0) {
        load(j, u);
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i)
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[e] = fmaf(w[i][e], win[i][e], y[e]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(w[TAPS - 1][e], u[e], y[e]);
#pragma unroll
        for (int i = 0; i + 1 < TAPS - 1; ++i)
#pragma unroll
          for (int e = 0; e < VEC; ++e) win[i][e] = win[i + 1][e];
        if (TAPS > 1) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) win[WIN - 1][e] = u[e];
        }
      } else {
        for (int i = 0; i < taps; ++i) {
          load(j - past + i, u);
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[e] = fmaf(a.w[static_cast<size_t>(i) * a.C + c0 + e], u[e], y[e]);
        }
      }
      const int p = pos0 + j;
      T* dst;
      if (c0 < a.nq) dst = static_cast<T*>(a.q) + static_cast<size_t>(r0 + j) * a.nq + c0;
      else {
        const int page = p / PGA_PAGE < a.page_ld ? a.pages[static_cast<size_t>(slot) * a.page_ld + p / PGA_PAGE] : -1;
        if (page < 0) {                                      // no page behind this position: nothing is written
          set_status(a.status, ST_BOUNDS, r0 + j, p, slot);
          continue;
        }
        const size_t tok = static_cast<size_t>(page) * PGA_PAGE + p % PGA_PAGE;
        dst = c0 < a.nq + a.nk ? static_cast<T*>(a.k) + tok * a.nk + (c0 - a.nq) : static_cast<T*>(a.v) + tok * a.nv + (c0 - a.nq - a.nk);
      }
#pragma unroll
      for (int i = 0; i < NV4; ++i) stf4(dst + 4 * i, make_float4(y[4 * i], y[4 * i + 1], y[4 * i + 2], y[4 * i + 3]));
    }
  }
  if (a.commit && blockIdx.x == 0) {
    const int m = a.n_rows ? min(n, a.n_rows[blockIdx.z]) : n;
    for (int i = 0; i < past && m > 0; ++i) {                // ascending: entry i is read before any later entry is written
      float u[VEC];
      load(m - past + i, u);
      T* d = tail + static_cast<size_t>(i) * a.C;
#pragma unroll
      for (int k = 0; k < NV4; ++k) stf4(d + 4 * k, make_float4(u[4 * k], u[4 * k + 1], u[4 * k + 2], u[4 * k + 3]));
    }
  }
}

// ------------------------------------------------------------------------------------------------ norm and rotation per head
struct HeadPrep {
  const void* proj;                      // [R, ldp]: H query heads, then G key heads (Dp columns each) and G value heads (Vp)
  const float *q_norm, *k_norm;          // [D] (null: no norm)
  void *q, *k, *v;                       // q [R, H * Dp]; caches as in PagedAttn
  const double* inv_freq;                // [rot / 2]
  const int *pos, *row_slot, *pages;
  int* status;
  double temp_every;
  int ldp, R, H, G, D, Dp, Vp, rot, page_ld;      // G 0: queries only
  float eps, temp_coef;
};

// grid (R, head groups); 256 threads: a warp per head, four consecutive channels per lane and step.
template <typename T>
__global__ void __launch_bounds__(256)
head_prep_kernel(const __grid_constant__ HeadPrep a) {
  extern __shared__ float2 turn[];                           // [rot / 2]: cosine and sine of the row's angles
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, lane = threadIdx.x & 31, p = a.pos[r];
  for (int i = threadIdx.x; i < a.rot / 2; i += 256) {
    float sn, cs;
    sincosf(static_cast<float>(static_cast<double>(p) * a.inv_freq[i]), &sn, &cs);
    turn[i] = make_float2(cs, sn);
  }
  __syncthreads();
  const T* row = static_cast<const T*>(a.proj) + static_cast<size_t>(r) * a.ldp;
  int page = 0;
  if (a.G > 0) {
    page = p / PGA_PAGE < a.page_ld ? a.pages[static_cast<size_t>(a.row_slot[r]) * a.page_ld + p / PGA_PAGE] : -1;
    if (page < 0 && threadIdx.x == 0 && blockIdx.y == 0) set_status(a.status, ST_BOUNDS, r, p, a.row_slot[r]);
  }
  const size_t tok = static_cast<size_t>(max(page, 0)) * PGA_PAGE + p % PGA_PAGE;
  for (int h = blockIdx.y * 8 + (threadIdx.x >> 5); h < a.H + 2 * a.G; h += gridDim.y * 8) {
    if (h >= a.H && page < 0) break;                         // no page behind this position: nothing is written
    if (h >= a.H + a.G) {
      const int g = h - a.H - a.G;
      const T* x = row + (a.H + a.G) * a.Dp + g * a.Vp;
      T* d = static_cast<T*>(a.v) + (tok * a.G + g) * a.Vp;
      for (int i = lane * 4; i < a.Vp; i += 128) stf4(d + i, ldf4(x + i));
      continue;
    }
    const bool isq = h < a.H;
    const T* x = row + h * a.Dp;
    T* d = isq ? static_cast<T*>(a.q) + (static_cast<size_t>(r) * a.H + h) * a.Dp : static_cast<T*>(a.k) + (tok * a.G + h - a.H) * a.Dp;
    const float* w = isq ? a.q_norm : a.k_norm;
    float4 x0 = make_float4(0.f, 0.f, 0.f, 0.f);             // (padded channels are zero)
    if (lane * 4 < a.Dp) x0 = ldf4(x + lane * 4);
    float m = 1.f;
    if (w) {
      float ss = x0.x * x0.x + x0.y * x0.y + x0.z * x0.z + x0.w * x0.w;
      for (int i = lane * 4 + 128; i < a.Dp; i += 128) { const float4 y = ldf4(x + i); ss += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w; }
      m = 1.f / sqrtf(warp_sum(ss) / a.D + a.eps);
    }
    if (isq && a.temp_coef != 0.f) m *= 1.f + a.temp_coef * logf(static_cast<float>(floor((p + 1) / a.temp_every)) + 1.f);
    for (int i = lane * 4; i < a.Dp; i += 128) {
      float4 y = i < 128 ? x0 : ldf4(x + i);
      if (w) {
        y.x *= i < a.D ? w[i] : 0.f; y.y *= i + 1 < a.D ? w[i + 1] : 0.f;
        y.z *= i + 2 < a.D ? w[i + 2] : 0.f; y.w *= i + 3 < a.D ? w[i + 3] : 0.f;
      }
      y.x *= m; y.y *= m; y.z *= m; y.w *= m;
      if (i < a.rot) { const float2 t = turn[i >> 1]; y = make_float4(y.x * t.x - y.y * t.y, y.y * t.x + y.x * t.y, y.z, y.w); }
      if (i + 2 < a.rot) { const float2 t = turn[(i >> 1) + 1]; y = make_float4(y.x, y.y, y.z * t.x - y.w * t.y, y.w * t.x + y.z * t.y); }
      stf4(d + i, y);
    }
  }
}

// ------------------------------------------------------------------------------------------------ one row, one head
// grid (rows, H); 128 threads.  V <= 1024.
template <typename T>
__global__ void __launch_bounds__(128)
paged_rows_kernel(const __grid_constant__ PagedAttn a) {
  extern __shared__ float sq[];                              // [D] query, then [128] weights
  __shared__ float sh[32];
  pdl_wait();
  const int h = blockIdx.y, t = threadIdx.x, pr = a.rows ? a.rows[blockIdx.x] : blockIdx.x, g = h / (a.H / a.G);
  float* sp = sq + a.D;
  for (int c = t; c < a.D; c += 128) sq[c] = ldf(static_cast<const T*>(a.q) + static_cast<size_t>(pr) * a.ldq + h * a.D + c);
  __syncthreads();
  const int p = a.pos[pr];
  const int* pg = a.pages + static_cast<size_t>(a.row_slot[pr]) * a.page_ld;
  auto token = [&](int tok) { return static_cast<size_t>(max(pg[tok / PGA_PAGE], 0)) * PGA_PAGE + tok % PGA_PAGE; };
  float acc[8];
#pragma unroll
  for (int c = 0; c < 8; ++c) acc[c] = 0.f;
  float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;
  for (int k0 = first_visible(p, a); k0 <= p; k0 += 128) {
    const int tok = k0 + t;
    float s = -INFINITY;
    if (tok <= p) {
      const T* row = static_cast<const T*>(a.k) + (token(tok) * a.G + g) * a.D;
      float x = 0.f;
      for (int c = 0; c < a.D; c += 4) {
        const float4 y = ldf4(row + c);
        x = fmaf(y.x, sq[c], x); x = fmaf(y.y, sq[c + 1], x); x = fmaf(y.z, sq[c + 2], x); x = fmaf(y.w, sq[c + 3], x);
      }
      s = x * a.scale;
      if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
      if (a.bias) s += a.bias[static_cast<size_t>(h) * a.bias_n + min(p - tok, a.bias_n - 1)];
      if (a.slopes) s -= a.slopes[h] * static_cast<float>(p - tok);
    }
    float mx = warp_max(s);
    if ((t & 31) == 0) sh[t >> 5] = mx;
    __syncthreads();
    mx = fmaxf(m, fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3])));
    const float e = tok <= p ? expf(s - mx) : 0.f, f = expf(m - mx);
    sp[t] = e;
    m = mx;
    __syncthreads();
    l = l * f + block_sum_all(e, sh);
    const int nt = min(128, p + 1 - k0);
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[c] *= f;
    for (int k = 0; k < nt; ++k) {
      const T* row = static_cast<const T*>(a.v) + (token(k0 + k) * a.G + g) * a.V;
      const float w = sp[k];
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (t + c * 128 < a.V) acc[c] = fmaf(w, ldf(row + t + c * 128), acc[c]);
    }
    __syncthreads();
  }
  const float inv = head_factor<T>(a, pr, h) / l;
#pragma unroll
  for (int c = 0; c < 8; ++c)
    if (t + c * 128 < a.V) stf(static_cast<T*>(a.out) + static_cast<size_t>(pr) * a.ldo + h * a.V + t + c * 128, acc[c] * inv);
}

// ------------------------------------------------------------------------------------------------ tensor-core helpers
__device__ __forceinline__ void pga_cp16(void* d, const void* s) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(d)), "l"(s) : "memory");
}
__device__ __forceinline__ void pga_ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void pga_ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void pga_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void pga_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// ------------------------------------------------------------------------------------------------ decode rows
constexpr int PGA_HEADS = 16;            // query heads per CTA (MMA rows)

// grid (rows, G * head groups, splits); 128 threads.  Split s covers page (page of the row's first visible key) + s.
__global__ void __launch_bounds__(128)
paged_decode_kernel(const __grid_constant__ PagedAttn a) {
  extern __shared__ __align__(16) uint8_t smem_pga[];
  const int D = a.D, V = a.V, LDK = D + 8, LDV = V + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_pga);      // [16][LDK]
  __nv_bfloat16* Ks = Qs + PGA_HEADS * LDK;                            // [64][LDK]
  __nv_bfloat16* Vs = Ks + PGA_PAGE * LDK;                             // [64][LDV]
  __nv_bfloat16* Ps = Vs + PGA_PAGE * LDV;                             // [2][16][72]: weights, high and low part
  float* Ss = reinterpret_cast<float*>(Ps + 2 * PGA_HEADS * 72);       // [16][68]
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, sp = blockIdx.z, pr = a.rows ? a.rows[r] : r;
  const int rep = a.H / a.G, groups = (rep + PGA_HEADS - 1) / PGA_HEADS, g = blockIdx.y / groups, hg = blockIdx.y % groups;
  const int h0 = g * rep + hg * PGA_HEADS, nh = min(PGA_HEADS, rep - hg * PGA_HEADS);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gg = lane >> 2, t = lane & 3;
  const int p = a.pos[pr], first = first_visible(p, a), page = first / PGA_PAGE + sp, k0 = page * PGA_PAGE;
  const size_t pb = (static_cast<size_t>(r) * a.H + h0) * a.nsplit + sp;
  if (k0 > p) {                                              // empty split
    if (tid < nh) {
      a.part_ml[(pb + static_cast<size_t>(tid) * a.nsplit) * 2] = -INFINITY;
      a.part_ml[(pb + static_cast<size_t>(tid) * a.nsplit) * 2 + 1] = 0.f;
    }
    return;
  }
  const int lo = max(first - k0, 0), hi = min(PGA_PAGE, p + 1 - k0);   // visible tokens of the page
  const size_t base = static_cast<size_t>(max(a.pages[static_cast<size_t>(a.row_slot[pr]) * a.page_ld + page], 0)) * PGA_PAGE;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(pr) * a.ldq + h0 * D;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(a.k) + (base * a.G + g) * D;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.v) + (base * a.G + g) * V;
  const int vk = D >> 3, vv = V >> 3;
  for (int i = tid; i < PGA_PAGE * vk; i += 128) {
    const int tok = i / vk, c = i - tok * vk;
    if (tok >= lo && tok < hi) pga_cp16(Ks + tok * LDK + c * 8, kc + static_cast<size_t>(tok) * a.G * D + c * 8);
    else *reinterpret_cast<uint4*>(Ks + tok * LDK + c * 8) = make_uint4(0u, 0u, 0u, 0u);
  }
  for (int i = tid; i < PGA_HEADS * vk; i += 128) {
    const int h = i / vk, c = i - h * vk;
    if (h < nh) pga_cp16(Qs + h * LDK + c * 8, q + h * D + c * 8);
    else *reinterpret_cast<uint4*>(Qs + h * LDK + c * 8) = make_uint4(0u, 0u, 0u, 0u);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int i = tid; i < PGA_PAGE * vv; i += 128) {
    const int tok = i / vv, c = i - tok * vv;
    if (tok >= lo && tok < hi) pga_cp16(Vs + tok * LDV + c * 8, vc + static_cast<size_t>(tok) * a.G * V + c * 8);
    else *reinterpret_cast<uint4*>(Vs + tok * LDV + c * 8) = make_uint4(0u, 0u, 0u, 0u);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  {                                                          // scores: warp w owns tokens [16w, 16w + 16)
    float s[2][4] = {};
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t x[4], b[4];
      pga_ldsm4(x, Qs + ((lane & 7) + ((lane >> 3) & 1) * 8) * LDK + ks * 16 + (lane >> 4) * 8);
      pga_ldsm4(b, Ks + (warp * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
      pga_mma(s[0], x, b[0], b[1]);
      pga_mma(s[1], x, b[2], b[3]);
    }
    const float icap = a.cap > 0.f ? 1.f / a.cap : 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = gg + (e >> 1) * 8, tok = warp * 16 + j * 8 + 2 * t + (e & 1);
        float x = -INFINITY;
        if (row < nh && tok >= lo && tok < hi) {
          x = s[j][e] * a.scale;
          if (a.cap > 0.f) x = a.cap * cap_tanh(x * icap);
          if (a.bias) x += __ldg(a.bias + static_cast<size_t>(h0 + row) * a.bias_n + min(p - k0 - tok, a.bias_n - 1));
          if (a.slopes) x -= __ldg(a.slopes + h0 + row) * static_cast<float>(p - k0 - tok);
        }
        Ss[row * 68 + tok] = x;
      }
  }
  __syncthreads();
  for (int row = warp; row < PGA_HEADS; row += 4) {          // softmax statistics of the page; a visible token exists
    const float s0 = Ss[row * 68 + lane], s1 = Ss[row * 68 + lane + 32];
    const float m = warp_max(fmaxf(s0, s1));
    const float e0 = s0 == -INFINITY ? 0.f : __expf(s0 - m), e1 = s1 == -INFINITY ? 0.f : __expf(s1 - m);
    const float l = warp_sum(e0 + e1);
    const __nv_bfloat16 b0 = __float2bfloat16(e0), b1 = __float2bfloat16(e1);
    Ps[row * 72 + lane] = b0;
    Ps[row * 72 + lane + 32] = b1;
    Ps[(PGA_HEADS + row) * 72 + lane] = __float2bfloat16(e0 - __bfloat162float(b0));
    Ps[(PGA_HEADS + row) * 72 + lane + 32] = __float2bfloat16(e1 - __bfloat162float(b1));
    if (lane == 0 && row < nh) {
      a.part_ml[(pb + static_cast<size_t>(row) * a.nsplit) * 2] = m;
      a.part_ml[(pb + static_cast<size_t>(row) * a.nsplit) * 2 + 1] = l;
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  for (int np = warp; np < V / 16; np += 4) {                // outputs: 16-wide column pairs round-robin over the warps
    float o[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < PGA_PAGE / 16; ++kk) {
      uint32_t b[4], x[4];
      pga_ldsm4t(b, Vs + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + np * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        pga_ldsm4(x, Ps + (half * PGA_HEADS + (lane & 7) + ((lane >> 3) & 1) * 8) * 72 + kk * 16 + (lane >> 4) * 8);
        pga_mma(o[0], x, b[0], b[1]);
        pga_mma(o[1], x, b[2], b[3]);
      }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int row = gg + hh * 8;
      if (row >= nh) continue;
      float* d = a.part_o + (pb + static_cast<size_t>(row) * a.nsplit) * V + np * 16 + 2 * t;
      *reinterpret_cast<float2*>(d) = make_float2(o[0][2 * hh], o[0][2 * hh + 1]);
      *reinterpret_cast<float2*>(d + 8) = make_float2(o[1][2 * hh], o[1][2 * hh + 1]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ prompts
// grid (row tiles, H, segments); NW warps x 16 rows.  VP >= V: compiled value width.  A key tile is one page.
template <int VP, int NW>
__global__ void __launch_bounds__(NW * 32, VP <= 64 ? 2 : 1)      // values of 128: two CTAs per SM spill and are 10 % slower
paged_prefill_kernel(const __grid_constant__ PagedAttn a) {
  constexpr int BM = NW * 16, BN = PGA_PAGE, LDV = VP + 8, NB = BM + BN;
  extern __shared__ __align__(16) uint8_t smem_pga[];
  const int D = a.D, LDK = D + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_pga);      // [BM][LDK]
  __nv_bfloat16* Ks = Qs + BM * LDK;                                   // [2][64][LDK]
  __nv_bfloat16* Vs = Ks + 2 * BN * LDK;                               // [2][64][LDV]
  float* Bs = reinterpret_cast<float*>(Vs + 2 * BN * LDV);             // [2][NB]: bias of the tile's distances, times log2 e
  const int* sg = a.segs + blockIdx.z * a.seg_ld;
  const int slot = sg[0], r0 = sg[1], n = sg[2], pos0 = sg[3], h = blockIdx.y, g = h / (a.H / a.G);
  const int qt = gridDim.x - 1 - blockIdx.x;                 // the longest row tiles first
  if (qt * BM >= n) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t = lane & 3;
  const int rows_valid = min(BM, n - qt * BM), pbase = pos0 + qt * BM;
  const int nkeys = pbase + rows_valid;
  const int j0 = first_visible(pbase, a) / BN, j1 = (nkeys + BN - 1) / BN;
  const int vk = D >> 3, vvs = a.V >> 3;
  constexpr int vv = VP >> 3;
  const int* pg = a.pages + static_cast<size_t>(slot) * a.page_ld;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(a.k) + static_cast<size_t>(g) * D;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.v) + static_cast<size_t>(g) * a.V;
  auto load_tile = [&](int j, int buf) {
    const size_t base = static_cast<size_t>(max(pg[j], 0)) * BN;
    const int valid = min(BN, nkeys - j * BN);
    __nv_bfloat16* kd = Ks + buf * BN * LDK;
    __nv_bfloat16* vd = Vs + buf * BN * LDV;
    for (int i = tid; i < BN * vk; i += NW * 32) {
      const int r = i / vk, c = i - r * vk;
      if (r < valid) pga_cp16(kd + r * LDK + c * 8, kc + (base + r) * a.G * D + c * 8);
      else *reinterpret_cast<uint4*>(kd + r * LDK + c * 8) = make_uint4(0u, 0u, 0u, 0u);
    }
    for (int i = tid; i < BN * vv; i += NW * 32) {
      const int r = i / vv, c = i - r * vv;
      if (r < valid && c < vvs) pga_cp16(vd + r * LDV + c * 8, vc + (base + r) * a.G * a.V + c * 8);
      else *reinterpret_cast<uint4*>(vd + r * LDV + c * 8) = make_uint4(0u, 0u, 0u, 0u);
    }
    if (a.bias)
      for (int i = tid; i < NB; i += NW * 32) {
        const int d = pbase - j * BN - (BN - 1) + i;
        Bs[buf * NB + i] = __ldg(a.bias + static_cast<size_t>(h) * a.bias_n + min(max(d, 0), a.bias_n - 1)) * PGA_LOG2E;
      }
  };
  for (int i = tid; i < BM * vk; i += NW * 32) {
    const int r = i / vk, c = i - r * vk, rr = min(r, rows_valid - 1);       // padded rows repeat the last valid row
    pga_cp16(Qs + r * LDK + c * 8, static_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(r0 + qt * BM + rr) * a.ldq + h * D + c * 8);
  }
  load_tile(j0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  float o[VP / 8][4];
#pragma unroll
  for (int i = 0; i < VP / 8; ++i) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
  // the sink is a key seen first: maximum = its score, sum = 1 (once per row: the quad's lane 0), output 0
  const float m0 = a.sink ? a.sink[h] * PGA_LOG2E : -INFINITY;
  float m_lo = m0, m_hi = m0, l_lo = a.sink && t == 0 ? 1.f : 0.f, l_hi = l_lo;
  const int w0 = pbase + warp * 16, p_lo = w0 + gq, p_hi = p_lo + 8;         // padded rows: positions past the segment, not stored
  const int f_lo = first_visible(p_lo, a), f_hi = first_visible(p_hi, a);
  const int w_first = first_visible(w0, a), w_last = first_visible(w0 + 15, a);
  const float slope = a.slopes ? a.slopes[h] * PGA_LOG2E : 0.f;
  const float qs = a.cap > 0.f ? a.scale / a.cap : a.scale * PGA_LOG2E, cs = a.cap * PGA_LOG2E, csqs = cs * qs;
  for (int j = j0; j < j1; ++j) {
    const int buf = (j - j0) & 1, k0 = j * BN;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (j + 1 < j1) { load_tile(j + 1, buf ^ 1); asm volatile("cp.async.commit_group;" ::: "memory"); }
    if (k0 > w0 + 15 || k0 + BN <= w_first) continue;        // no row of this warp sees the tile
    const __nv_bfloat16* kb = Ks + buf * BN * LDK;
    const __nv_bfloat16* vb = Vs + buf * BN * LDV;
    const float* bs = Bs + buf * NB + warp * 16 + gq + 8 - 2 * t + (BN - 1);   // distance of row p_hi and key k0 + 2t
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) { s[i][0] = 0.f; s[i][1] = 0.f; s[i][2] = 0.f; s[i][3] = 0.f; }
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t x[4];
      pga_ldsm4(x, Qs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + ks * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        pga_ldsm4(b, kb + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
        pga_mma(s[2 * np], x, b[0], b[1]);
        pga_mma(s[2 * np + 1], x, b[2], b[3]);
      }
    }
    const bool need_mask = k0 + BN - 1 > w0 || k0 < w_last;
    if (a.cap > 0.f) {                                       // one form for the whole tile: scores far below the cap need no exponential
      float big = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) big = fmaxf(big, fmaxf(fmaxf(fabsf(s[i][0]), fabsf(s[i][1])), fmaxf(fabsf(s[i][2]), fabsf(s[i][3]))));
      if (__any_sync(0xffffffffu, big * fabsf(qs) >= CAP_NEAR)) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][e] = cs * cap_tanh(s[i][e] * qs);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][e] *= csqs * tanh_over_z(s[i][e] * qs);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] *= qs;
    }
    if (a.slopes) {
      const float d = static_cast<float>(k0 + 2 * t - p_lo);
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] = fmaf(slope, d + static_cast<float>(i * 8 + (e & 1) - (e >> 1) * 8), s[i][e]);
    }
    float mx_lo = m_lo, mx_hi = m_hi;
    float b_hi[2] = {0.f, 0.f}, b_lo[2] = {0.f, 0.f};
    if (a.bias) { b_lo[0] = bs[0]; b_lo[1] = bs[-1]; }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      // bias depends on the distance only: keys i * 8 of row p_lo are as far as keys (i + 1) * 8 of row p_hi
      if (a.bias) { b_hi[0] = b_lo[0]; b_hi[1] = b_lo[1]; b_lo[0] = bs[-8 * i - 8]; b_lo[1] = bs[-8 * i - 9]; }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = s[i][e] + ((e >> 1) ? b_hi[e & 1] : b_lo[e & 1]);
        if (need_mask) {
          const int key = k0 + i * 8 + 2 * t + (e & 1);
          if (key > ((e >> 1) ? p_hi : p_lo) || key < ((e >> 1) ? f_hi : f_lo)) v = -INFINITY;
        }
        s[i][e] = v;
      }
      mx_lo = fmaxf(mx_lo, fmaxf(s[i][0], s[i][1]));
      mx_hi = fmaxf(mx_hi, fmaxf(s[i][2], s[i][3]));
    }
    mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1)); mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
    mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1)); mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
    // without a sink a row may have seen no key yet: exponentials are then taken against 0 and every term stays 0
    const float z_lo = mx_lo == -INFINITY ? 0.f : mx_lo, z_hi = mx_hi == -INFINITY ? 0.f : mx_hi;
    const float c_lo = exp2f(m_lo - z_lo), c_hi = exp2f(m_hi - z_hi);
    m_lo = mx_lo; m_hi = mx_hi;
    float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      s[i][0] = exp2f(s[i][0] - z_lo); s[i][1] = exp2f(s[i][1] - z_lo);
      s[i][2] = exp2f(s[i][2] - z_hi); s[i][3] = exp2f(s[i][3] - z_hi);
      sum_lo += s[i][0] + s[i][1]; sum_hi += s[i][2] + s[i][3];
    }
    l_lo = l_lo * c_lo + sum_lo; l_hi = l_hi * c_hi + sum_hi;
#pragma unroll
    for (int i = 0; i < VP / 8; ++i) { o[i][0] *= c_lo; o[i][1] *= c_lo; o[i][2] *= c_hi; o[i][3] *= c_hi; }
#pragma unroll
    for (int kk = 0; kk < BN / 16; ++kk) {
      uint32_t ph[4], pl[4];
      pga_split2(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]); pga_split2(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
      pga_split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]); pga_split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
      for (int np = 0; np < VP / 16; ++np) {
        uint32_t b[4];
        pga_ldsm4t(b, vb + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + np * 16 + (lane >> 4) * 8);
        pga_mma(o[2 * np], ph, b[0], b[1]); pga_mma(o[2 * np + 1], ph, b[2], b[3]);
        pga_mma(o[2 * np], pl, b[0], b[1]); pga_mma(o[2 * np + 1], pl, b[2], b[3]);
      }
    }
  }
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int rl = warp * 16 + gq + hh * 8;
    if (rl >= rows_valid) continue;
    const float inv = head_factor<__nv_bfloat16>(a, r0 + qt * BM + rl, h) / (hh ? l_hi : l_lo);
    __nv_bfloat16* d = static_cast<__nv_bfloat16*>(a.out) + static_cast<size_t>(r0 + qt * BM + rl) * a.ldo + h * a.V + 2 * t;
#pragma unroll
    for (int i = 0; i < VP / 8; ++i)
      if (i * 8 < a.V) *reinterpret_cast<__nv_bfloat162*>(d + i * 8) = __floats2bfloat162_rn(o[i][2 * hh] * inv, o[i][2 * hh + 1] * inv);
  }
}

constexpr int PGA_SMEM = 220 * 1024;

template <int VP, int NW>
static int launch_paged_prefill(const PagedAttn& a, int nseg, int max_rows, cudaStream_t s) {
  auto kern = paged_prefill_kernel<VP, NW>;
  const int smem = ((NW * 16 + 2 * PGA_PAGE) * (a.D + 8) + 2 * PGA_PAGE * (VP + 8)) * 2 + 2 * (NW * 16 + PGA_PAGE) * 4;
  if (smem > PGA_SMEM) return -6;
  static bool done = false;
  if (!done) { cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, PGA_SMEM); done = true; }
  kern<<<dim3((max_rows + NW * 16 - 1) / (NW * 16), a.H, nseg), NW * 32, smem, s>>>(a);
  return spark_launch_rc("spark_paged_prefill");
}

static bool paged_ok(const PagedAttn* a) {
  return a->H > 0 && a->G > 0 && a->H % a->G == 0 && a->D > 0 && a->V > 0 && ((a->D | a->V) & 15) == 0 && (a->ldq & 7) == 0 &&
         (!a->bias || a->bias_n > 0) && (a->ldo & 3) == 0 && a->ldo >= a->H * a->V;
}

}  // namespace spark

using namespace spark;

// Rows of all segments: convolution, cache rows (store) and the advanced tails (commit; by n_rows[i] rows if given).
extern "C" int spark_conv_prep(const ConvPrep* a, int nseg, int max_rows, int f32, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  if (a->taps < 1 || ((a->C | a->nq | a->nk | a->nv | a->ldp) & 7) || a->C != a->nq + a->nk + a->nv) return -5;
  ConvPrep c = *a;
  c.tile = max_rows <= 16 ? 16 : 32;
  if (c.tile < a->taps - 1) c.tile = a->taps - 1;
  const int vec = f32 ? 4 : 8;
  const dim3 grid(a->store ? (max_rows + c.tile - 1) / c.tile : 1, (a->C / vec + 127) / 128, nseg);
#define SPARK_CONV(T, TAPS) spark_launch_pdl(conv_prep_kernel<T, TAPS>, grid, dim3(128), 0, s, dim3(1, 1, 1), c)
#define SPARK_CONV_T(T)               \
  if (a->taps == 2) SPARK_CONV(T, 2); \
  else if (a->taps == 3) SPARK_CONV(T, 3); \
  else if (a->taps == 4) SPARK_CONV(T, 4); \
  else SPARK_CONV(T, 0);
  if (f32) { SPARK_CONV_T(float) } else { SPARK_CONV_T(__nv_bfloat16) }
#undef SPARK_CONV_T
#undef SPARK_CONV
  return spark_launch_rc(__func__);
}

// Rows of the whole plan: finished queries, and with G > 0 the cache rows.
extern "C" int spark_head_prep(const HeadPrep* a, int f32, cudaStream_t s) {
  if (a->R <= 0) return 0;
  if (a->H <= 0 || ((a->Dp | a->Vp) & 15) || a->D > a->Dp || (a->rot & 1) || a->rot > a->D || (a->ldp & 7) || a->rot > 8192 ||
      a->ldp < a->H * a->Dp + a->G * (a->Dp + a->Vp) || (a->rot && !a->inv_freq) || !(a->temp_every > 0.0)) return -5;
  const int groups = (a->H + 2 * a->G + 7) / 8;
  const dim3 grid(a->R, a->R <= 128 && groups <= 65535 ? groups : 1);    // few rows: a head per warp
  if (f32) spark_launch_pdl(head_prep_kernel<float>, grid, dim3(256), a->rot * 4, s, dim3(1, 1, 1), *a);
  else spark_launch_pdl(head_prep_kernel<__nv_bfloat16>, grid, dim3(256), a->rot * 4, s, dim3(1, 1, 1), *a);
  return spark_launch_rc(__func__);
}

extern "C" int spark_paged_rows(const PagedAttn* a, int n, int f32, cudaStream_t s) {
  if (n <= 0) return 0;
  if (!paged_ok(a) || a->V > 1024 || a->D > 8192 || a->H > 65535) return -5;
  const size_t smem = (a->D + 128) * 4;
  if (f32) spark_launch_pdl(paged_rows_kernel<float>, dim3(n, a->H), dim3(128), smem, s, dim3(1, 1, 1), *a);
  else spark_launch_pdl(paged_rows_kernel<__nv_bfloat16>, dim3(n, a->H), dim3(128), smem, s, dim3(1, 1, 1), *a);
  return spark_launch_rc(__func__);
}

// bf16.  part_o fp32 [n, H, nsplit, V], part_ml fp32 [n, H, nsplit, 2]; nsplit >= pages that any row's visible keys span.
extern "C" int spark_paged_decode(const PagedAttn* a, int n, cudaStream_t s) {
  if (n <= 0) return 0;
  if (!paged_ok(a) || a->nsplit <= 0 || a->nsplit > 65535) return -5;
  const int smem = ((PGA_HEADS + PGA_PAGE) * (a->D + 8) + PGA_PAGE * (a->V + 8) + 2 * PGA_HEADS * 72) * 2 + PGA_HEADS * 68 * 4;
  if (smem > PGA_SMEM) return -6;
  static bool done = false;
  if (!done) { cudaFuncSetAttribute(paged_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, PGA_SMEM); done = true; }
  const int rep = a->H / a->G, groups = (rep + PGA_HEADS - 1) / PGA_HEADS;
  if (a->G * groups > 65535) return -5;
  spark_launch_pdl(paged_decode_kernel, dim3(n, a->G * groups, a->nsplit), dim3(128), smem, s, dim3(1, 1, 1), *a);
  const int rc = launch_split_merge(a->part_o, a->part_ml, a->nsplit, a->sink, n, a->H, a->V, a->out, a->gate, a->ldg, a->rows, 1, s, a->ldo, a->out_scale);
  return rc ? rc : spark_launch_rc(__func__);
}

// bf16.  -6: the head sizes do not fit shared memory (the caller uses spark_paged_rows).
extern "C" int spark_paged_prefill(const PagedAttn* a, int nseg, int max_rows, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  if (!paged_ok(a) || a->H > 65535 || nseg > 65535) return -5;
  if (a->V <= 32) return launch_paged_prefill<32, 8>(*a, nseg, max_rows, s);
  if (a->V <= 64) return launch_paged_prefill<64, 8>(*a, nseg, max_rows, s);
  if (a->V <= 128) return launch_paged_prefill<128, 8>(*a, nseg, max_rows, s);
  if (a->V <= 256) return launch_paged_prefill<256, 8>(*a, nseg, max_rows, s);
  return -6;
}
