// Dense causal latent attention over a paged cache (64-token pages of [latent | rotated key] rows), for bf16 and fp32
// activations.  Decode rows run in the absorbed form (mla.cu, `spark_mla_attn_paged`); this file holds
//
//   latent_prep      per row: RMSNorm of the query latent, RMSNorm of the key/value latent, rotation of the shared key part,
//                    and the cache row written to its page
//   latent_qrope     rotation of the queries' rotated part, in place or into the tail of absorbed query rows
//   latent_gather    the pages of a sequence as contiguous rows (operand of the key / value up-projection of prompts)
//   latent_prefill   prompts: flash-style attention on the up-projected keys and values; scores, softmax and its weights in
//                    fp32 (the weights enter the second product as two-term bf16 sums)
//   latent_rows      one CTA per (row, head) in the absorbed form on the FP32 units: the 32-bit mode, and shapes the
//                    tensor-core kernels do not cover
// Rotary pairs are (2i, 2i + 1) when `interleaved`, else (i, i + rope/2).  Queries may come straight from the projected row (no
// query latent) and rows may have no rotated part.  An optional sink per head enters the denominator only; the output gate is one
// sigmoid per head, or per element of the concatenated heads (prompts here; absorbed rows: in the product behind the attention).
#include "../common/rows.cuh"

namespace spark {

constexpr int LAT_PAGE = 64;

struct LatentShape {
  int q_rank, ldcq, L, Lp, rope, Rp;        // Lp / Rp: padded widths of the two parts of a cache row
  int interleaved;
  float eps;
};

__device__ __forceinline__ void rope_pair(int i, int rope, int interleaved, int& a, int& b) {
  a = interleaved ? 2 * i : i;
  b = interleaved ? 2 * i + 1 : (rope >> 1) + i;
}
__device__ __forceinline__ void rope_sincos(int pos, double inv, float& sn, float& cs) {
  sincosf(static_cast<float>(static_cast<double>(pos) * inv), &sn, &cs);
}

// grid R; 128 threads.  proj: [R, ldp], the query latent at column oq, the key/value latent at okv, the key part at okr.
template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const T* __restrict__ proj, int ldp, int oq, int okv, int okr, LatentShape d, const float* __restrict__ q_norm,
                   const float* __restrict__ kv_norm, const double* __restrict__ inv_freq, const int* __restrict__ pos,
                   const int* __restrict__ row_slot, const int* __restrict__ pages, int page_ld, T* __restrict__ cq,
                   T* __restrict__ cache, int* __restrict__ status) {
  __shared__ float sh[32];
  pdl_wait();
  const int r = blockIdx.x, t = threadIdx.x, p = pos[r];
  const T* a = proj + static_cast<size_t>(r) * ldp;
  float ss = 0.f, rs;
  if (d.q_rank > 0) {
    for (int i = t; i < d.q_rank; i += 128) { const float x = ldf(a + oq + i); ss = fmaf(x, x, ss); }
    rs = 1.f / sqrtf(block_sum_all(ss, sh) / d.q_rank + d.eps);
    for (int i = t; i < d.ldcq; i += 128)
      stf(cq + static_cast<size_t>(r) * d.ldcq + i, i < d.q_rank ? ldf(a + oq + i) * rs * q_norm[i] : 0.f);
    ss = 0.f;
  }
  for (int i = t; i < d.L; i += 128) { const float x = ldf(a + okv + i); ss = fmaf(x, x, ss); }
  rs = 1.f / sqrtf(block_sum_all(ss, sh) / d.L + d.eps);
  const int page = p / LAT_PAGE < page_ld ? pages[static_cast<size_t>(row_slot[r]) * page_ld + p / LAT_PAGE] : -1;
  if (page < 0) {                                           // no page behind this position: nothing is written
    if (t == 0) set_status(status, ST_BOUNDS, r, p, row_slot[r]);
    return;
  }
  T* row = cache + (static_cast<size_t>(page) * LAT_PAGE + p % LAT_PAGE) * (d.Lp + d.Rp);
  for (int i = t; i < d.Lp; i += 128) stf(row + i, i < d.L ? ldf(a + okv + i) * rs * kv_norm[i] : 0.f);
  for (int i = t; i < d.Rp - d.rope; i += 128) stf(row + d.Lp + d.rope + i, 0.f);
  for (int i = t; i < d.rope / 2; i += 128) {
    int u, v;
    rope_pair(i, d.rope, d.interleaved, u, v);
    float sn, cs;
    rope_sincos(p, inv_freq[i], sn, cs);
    const float x = ldf(a + okr + u), y = ldf(a + okr + v);
    stf(row + d.Lp + u, x * cs - y * sn);
    stf(row + d.Lp + v, y * cs + x * sn);
  }
}

// grid (rows, ceil(H * Rp / 2 / 128)).  src: plan rows [.., lds], head h's rotated part at h * hss; dst row i at i * ldd + h * hsd.
template <typename T>
__global__ void __launch_bounds__(128)
latent_qrope_kernel(const T* __restrict__ src, int lds, int hss, T* __restrict__ dst, int ldd, int hsd, int H, int rope, int Rp,
                    int interleaved, const double* __restrict__ inv_freq, const int* __restrict__ pos, const int* __restrict__ rows,
                    int src_compact) {
  pdl_wait();
  const int i = blockIdx.x, pr = rows ? rows[i] : i, j = blockIdx.y * 128 + threadIdx.x, half = Rp / 2;
  if (j >= H * half) return;
  const int h = j / half, k = j - h * half;
  const T* s = src + static_cast<size_t>(src_compact ? i : pr) * lds + h * hss;
  T* o = dst + static_cast<size_t>(i) * ldd + h * hsd;
  if (k >= rope / 2) { stf(o + 2 * k, 0.f); stf(o + 2 * k + 1, 0.f); return; }     // padding behind the rotated part
  int u, v;
  rope_pair(k, rope, interleaved, u, v);
  float sn, cs;
  rope_sincos(pos[pr], inv_freq[k], sn, cs);
  const float x = ldf(s + u), y = ldf(s + v);
  stf(o + u, x * cs - y * sn);
  stf(o + v, y * cs + x * sn);
}

// segs: [n][5] = slot, first plan row, rows, first position, first gathered row.  grid (tokens / 8, n); 256 threads.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, int vec, const int* __restrict__ segs, const int* __restrict__ pages, int page_ld,
                     uint4* __restrict__ out) {
  const int* sg = segs + blockIdx.y * 5;
  const int ctx = sg[3] + sg[2], tok = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (tok >= ctx) return;
  const int page = max(pages[static_cast<size_t>(sg[0]) * page_ld + tok / LAT_PAGE], 0);
  const uint4* s = cache + (static_cast<size_t>(page) * LAT_PAGE + tok % LAT_PAGE) * vec;
  uint4* d = out + (static_cast<size_t>(sg[4]) + tok) * vec;
  for (int i = threadIdx.x & 31; i < vec; i += 32) d[i] = s[i];
}

// ------------------------------------------------------------------------------------------------ one row, one head
// grid (rows, H); 128 threads.  q_full [n, H, KW] (absorbed latent part | rotated part), out [n, H, Lp].
template <typename T>
__global__ void __launch_bounds__(128)
latent_rows_kernel(const T* __restrict__ q_full, const T* __restrict__ cache, const int* __restrict__ pos, const int* __restrict__ rows,
                   const int* __restrict__ row_slot, const int* __restrict__ pages, int page_ld, int H, int Lp, int Rp, float scale,
                   const T* __restrict__ gate, int ldg, const float* __restrict__ sink, T* __restrict__ out) {
  extern __shared__ float sq[];                              // [KW] query, then [128] weights
  __shared__ float sh[32];
  pdl_wait();
  const int i = blockIdx.x, h = blockIdx.y, t = threadIdx.x, pr = rows ? rows[i] : i, KW = Lp + Rp;
  float* sp = sq + KW;
  for (int c = t; c < KW; c += 128) sq[c] = ldf(q_full + (static_cast<size_t>(i) * H + h) * KW + c);
  __syncthreads();
  const int n = pos[pr] + 1;
  const int* pg = pages + static_cast<size_t>(row_slot[pr]) * page_ld;
  float acc[8];
#pragma unroll
  for (int c = 0; c < 8; ++c) acc[c] = 0.f;
  float m = sink ? sink[h] : -INFINITY, l = sink ? 1.f : 0.f;
  for (int k0 = 0; k0 < n; k0 += 128) {
    const int tok = k0 + t;
    float s = -INFINITY;
    if (tok < n) {
      const T* row = cache + (static_cast<size_t>(max(pg[tok / LAT_PAGE], 0)) * LAT_PAGE + tok % LAT_PAGE) * KW;
      float a = 0.f;
      for (int c = 0; c < KW; c += 4) {
        const float4 x = ldf4(row + c);
        a = fmaf(x.x, sq[c], a); a = fmaf(x.y, sq[c + 1], a); a = fmaf(x.z, sq[c + 2], a); a = fmaf(x.w, sq[c + 3], a);
      }
      s = a * scale;
    }
    float mx = warp_max(s);
    if ((t & 31) == 0) sh[t >> 5] = mx;
    __syncthreads();
    mx = fmaxf(m, fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3])));
    const float e = tok < n ? expf(s - mx) : 0.f, f = expf(m - mx);
    sp[t] = e;
    m = mx;
    __syncthreads();
    l = l * f + block_sum_all(e, sh);
    const int nt = min(128, n - k0);
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[c] *= f;
    for (int k = 0; k < nt; ++k) {
      const int tk = k0 + k;
      const T* row = cache + (static_cast<size_t>(max(pg[tk / LAT_PAGE], 0)) * LAT_PAGE + tk % LAT_PAGE) * KW;
      const float p = sp[k];
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (t + c * 128 < Lp) acc[c] = fmaf(p, ldf(row + t + c * 128), acc[c]);
    }
    __syncthreads();
  }
  float inv = 1.f / l;
  if (gate) inv *= sigmoid_f(ldf(gate + static_cast<size_t>(pr) * ldg + h));
#pragma unroll
  for (int c = 0; c < 8; ++c)
    if (t + c * 128 < Lp) stf(out + (static_cast<size_t>(i) * H + h) * Lp + t + c * 128, acc[c] * inv);
}

// ------------------------------------------------------------------------------------------------ prompts
constexpr int LPF_BN = 64;

__device__ __forceinline__ void lp_cp16(void* d, const void* s) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(d)), "l"(s) : "memory");
}
__device__ __forceinline__ void lp_ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lp_ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lp_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lp_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct LatentPrefill {
  const __nv_bfloat16 *q, *kv, *lat, *gate;
  __nv_bfloat16* out;
  const int* segs;                 // [n][5]
  const float* sink;               // [H]
  int ldq, ldkv, ldlat, ldg, ldo, H, Dp, Rp, V, Vp, Lp, gate_all;      // gate_all: a gate column per output column, else per head
  float scale_log2;
};

// grid (row tiles, H, segments); NW warps x 16 rows.  q rows hold [Dp | Rp] per head, kv rows [Dp | Vp] per head, lat rows the
// rotated key part at column Lp.  VP >= Vp: compiled value width.
template <int VP, int NW>
__global__ void __launch_bounds__(NW * 32)
latent_prefill_kernel(const __grid_constant__ LatentPrefill a) {
  constexpr int BM = NW * 16, LDV = VP + 8;
  extern __shared__ __align__(16) uint8_t smem_lp[];
  const int KD = a.Dp + a.Rp, LDK = KD + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_lp);       // [BM][LDK]
  __nv_bfloat16* Ks = Qs + BM * LDK;                                     // [2][64][LDK]
  __nv_bfloat16* Vs = Ks + 2 * LPF_BN * LDK;                             // [2][64][LDV]
  const int* sg = a.segs + blockIdx.z * 5;
  const int r0 = sg[1], n = sg[2], pos0 = sg[3], c0 = sg[4], h = blockIdx.y;
  const int qt = gridDim.x - 1 - blockIdx.x;                 // the longest row tiles first
  if (qt * BM >= n) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int rows_valid = min(BM, n - qt * BM);
  const int nkeys = pos0 + qt * BM + rows_valid, ntiles = (nkeys + LPF_BN - 1) / LPF_BN;
  const int vk = KD >> 3, vd = a.Dp >> 3, vv = VP >> 3, vvs = a.Vp >> 3;
  auto load_kv = [&](int j, int buf) {
    __nv_bfloat16* kd = Ks + buf * LPF_BN * LDK;
    __nv_bfloat16* vdst = Vs + buf * LPF_BN * LDV;
    for (int i = tid; i < LPF_BN * vk; i += NW * 32) {
      const int r = i / vk, c = i - r * vk, key = j * LPF_BN + r;
      __nv_bfloat16* d = kd + r * LDK + c * 8;
      if (key < nkeys) {
        const size_t row = static_cast<size_t>(c0) + key;
        lp_cp16(d, c < vd ? a.kv + row * a.ldkv + h * (a.Dp + a.Vp) + c * 8 : a.lat + row * a.ldlat + a.Lp + (c - vd) * 8);
      } else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
    for (int i = tid; i < LPF_BN * vv; i += NW * 32) {
      const int r = i / vv, c = i - r * vv, key = j * LPF_BN + r;
      __nv_bfloat16* d = vdst + r * LDV + c * 8;
      if (key < nkeys && c < vvs) lp_cp16(d, a.kv + (static_cast<size_t>(c0) + key) * a.ldkv + h * (a.Dp + a.Vp) + a.Dp + c * 8);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
  };
  for (int i = tid; i < BM * vk; i += NW * 32) {
    const int r = i / vk, c = i - r * vk, rr = min(r, rows_valid - 1);       // padded rows repeat the last valid row
    lp_cp16(Qs + r * LDK + c * 8, a.q + static_cast<size_t>(r0 + qt * BM + rr) * a.ldq + h * KD + c * 8);
  }
  load_kv(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  float o[VP / 8][4];
#pragma unroll
  for (int i = 0; i < VP / 8; ++i) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
  // the sink is a key seen first: maximum = its score, sum = 1 (once per row: the quad's lane 0), output 0
  const float m0 = a.sink ? a.sink[h] * 1.4426950408889634f : -INFINITY;
  float m_lo = m0, m_hi = m0, l_lo = a.sink && t == 0 ? 1.f : 0.f, l_hi = l_lo;
  const int p_lo = pos0 + qt * BM + min(warp * 16 + g, rows_valid - 1);
  const int p_hi = pos0 + qt * BM + min(warp * 16 + g + 8, rows_valid - 1);
  const int p_first = pos0 + qt * BM + min(warp * 16, rows_valid - 1);
  const int p_last = pos0 + qt * BM + min(warp * 16 + 15, rows_valid - 1);
  for (int j = 0; j < ntiles; ++j) {
    const int buf = j & 1, k0 = j * LPF_BN;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (j + 1 < ntiles) { load_kv(j + 1, buf ^ 1); asm volatile("cp.async.commit_group;" ::: "memory"); }
    if (k0 > p_last) continue;                                // no row of this warp sees the tile
    const __nv_bfloat16* kb = Ks + buf * LPF_BN * LDK;
    const __nv_bfloat16* vb = Vs + buf * LPF_BN * LDV;
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) { s[i][0] = 0.f; s[i][1] = 0.f; s[i][2] = 0.f; s[i][3] = 0.f; }
    for (int ks = 0; ks < KD / 16; ++ks) {
      uint32_t x[4];
      lp_ldsm4(x, Qs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + ks * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        lp_ldsm4(b, kb + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
        lp_mma(s[2 * np], x, b[0], b[1]);
        lp_mma(s[2 * np + 1], x, b[2], b[3]);
      }
    }
    const bool need_mask = k0 + LPF_BN - 1 > p_first;
    float mx_lo = m_lo, mx_hi = m_hi;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = s[i][e] * a.scale_log2;
        if (need_mask && k0 + i * 8 + 2 * t + (e & 1) > ((e >> 1) ? p_hi : p_lo)) v = -INFINITY;
        s[i][e] = v;
      }
      mx_lo = fmaxf(mx_lo, fmaxf(s[i][0], s[i][1]));
      mx_hi = fmaxf(mx_hi, fmaxf(s[i][2], s[i][3]));
    }
    mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1)); mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
    mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1)); mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
    // key 0 is in the first tile and visible to every row, so the running maxima are finite from there on
    const float f_lo = exp2f(m_lo - mx_lo), f_hi = exp2f(m_hi - mx_hi);
    m_lo = mx_lo; m_hi = mx_hi;
    float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      s[i][0] = exp2f(s[i][0] - mx_lo); s[i][1] = exp2f(s[i][1] - mx_lo);
      s[i][2] = exp2f(s[i][2] - mx_hi); s[i][3] = exp2f(s[i][3] - mx_hi);
      sum_lo += s[i][0] + s[i][1]; sum_hi += s[i][2] + s[i][3];
    }
    l_lo = l_lo * f_lo + sum_lo; l_hi = l_hi * f_hi + sum_hi;
#pragma unroll
    for (int i = 0; i < VP / 8; ++i) { o[i][0] *= f_lo; o[i][1] *= f_lo; o[i][2] *= f_hi; o[i][3] *= f_hi; }
#pragma unroll
    for (int kk = 0; kk < LPF_BN / 16; ++kk) {
      uint32_t ph[4], pl[4];
      lp_split2(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]); lp_split2(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
      lp_split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]); lp_split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
      for (int np = 0; np < VP / 16; ++np) {
        uint32_t b[4];
        lp_ldsm4t(b, vb + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + np * 16 + (lane >> 4) * 8);
        lp_mma(o[2 * np], ph, b[0], b[1]); lp_mma(o[2 * np + 1], ph, b[2], b[3]);
        lp_mma(o[2 * np], pl, b[0], b[1]); lp_mma(o[2 * np + 1], pl, b[2], b[3]);
      }
    }
  }
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int rl = warp * 16 + g + hh * 8;
    if (rl >= rows_valid) continue;
    const size_t r = static_cast<size_t>(r0 + qt * BM + rl);
    float inv = 1.f / (hh ? l_hi : l_lo);
    const __nv_bfloat16* gate = a.gate ? a.gate + r * a.ldg + (a.gate_all ? h * a.V : h) : nullptr;
    if (gate && !a.gate_all) inv *= sigmoid_f(__bfloat162float(*gate));
    const bool each = gate && a.gate_all;
    __nv_bfloat16* o_row = a.out + r * a.ldo + h * a.V;
    if (((a.V | a.ldo | (each ? a.ldg : 0)) & 1) == 0) {       // column pairs are 4-byte aligned
#pragma unroll
      for (int i = 0; i < VP / 8; ++i) {
        const int d = i * 8 + 2 * t;
        if (d >= a.V) continue;
        float x = o[i][2 * hh] * inv, y = o[i][2 * hh + 1] * inv;
        if (each) {
          const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + d));
          x *= sigmoid_t<__nv_bfloat16>(g.x); y *= sigmoid_t<__nv_bfloat16>(g.y);
        }
        *reinterpret_cast<__nv_bfloat162*>(o_row + d) = __floats2bfloat162_rn(x, y);
      }
      continue;
    }
#pragma unroll
    for (int i = 0; i < VP / 8; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = i * 8 + 2 * t + e;
        if (d >= a.V) continue;
        const float x = o[i][2 * hh + e] * inv;
        o_row[d] = __float2bfloat16(each ? x * sigmoid_t<__nv_bfloat16>(__bfloat162float(gate[d])) : x);
      }
  }
}

template <int VP, int NW>
static int launch_latent_prefill(const LatentPrefill& a, int nseg, int max_rows, cudaStream_t s) {
  auto kern = latent_prefill_kernel<VP, NW>;
  const int LDK = a.Dp + a.Rp + 8;
  const int smem = ((NW * 16 + 2 * LPF_BN) * LDK + 2 * LPF_BN * (VP + 8)) * 2;
  if (smem > 220 * 1024) return -6;
  static bool done = false;
  if (!done) { cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024); done = true; }
  kern<<<dim3((max_rows + NW * 16 - 1) / (NW * 16), a.H, nseg), NW * 32, smem, s>>>(a);
  return spark_launch_rc("spark_latent_prefill");
}

}  // namespace spark

using namespace spark;

#define SPARK_BY_TYPE(f32, CALL)          \
  if (f32) { using T = float; CALL; }     \
  else { using T = __nv_bfloat16; CALL; }

extern "C" int spark_latent_prep(const void* proj, int ldp, int oq, int okv, int okr, int R, int q_rank, int ldcq, int L, int Lp,
                                 int rope, int Rp, int interleaved, float eps, const float* q_norm, const float* kv_norm,
                                 const double* inv_freq, const int* pos, const int* row_slot, const int* pages, int page_ld, void* cq,
                                 void* cache, int f32, int* status, cudaStream_t s) {
  if (R <= 0) return 0;
  if (rope & 1 || Rp & 1 || Rp < rope || Lp < L) return -5;
  const LatentShape d{q_rank, ldcq, L, Lp, rope, Rp, interleaved, eps};
  SPARK_BY_TYPE(f32, spark_launch_pdl(latent_prep_kernel<T>, dim3(R), dim3(128), 0, s, dim3(1, 1, 1), (const T*)proj, ldp, oq, okv, okr,
                                      d, q_norm, kv_norm, inv_freq, pos, row_slot, pages, page_ld, (T*)cq, (T*)cache, status))
  return spark_launch_rc(__func__);
}

extern "C" int spark_latent_qrope(const void* src, int lds, int hss, void* dst, int ldd, int hsd, int n, int H, int rope, int Rp,
                                  int interleaved, const double* inv_freq, const int* pos, const int* rows, int src_compact, int f32,
                                  cudaStream_t s) {
  if (n <= 0 || Rp <= 0) return 0;
  SPARK_BY_TYPE(f32, spark_launch_pdl(latent_qrope_kernel<T>, dim3(n, (H * (Rp / 2) + 127) / 128), dim3(128), 0, s, dim3(1, 1, 1),
                                      (const T*)src, lds, hss, (T*)dst, ldd, hsd, H, rope, Rp, interleaved, inv_freq, pos, rows,
                                      src_compact))
  return spark_launch_rc(__func__);
}

// width: bytes of a cache row (multiple of 16).
extern "C" int spark_latent_gather(const void* cache, int width, const int* segs, int nseg, int max_ctx, const int* pages, int page_ld,
                                   void* out, cudaStream_t s) {
  if (nseg <= 0) return 0;
  if (width & 15) return -5;
  latent_gather_kernel<<<dim3((max_ctx + 7) / 8, nseg), 256, 0, s>>>((const uint4*)cache, width / 16, segs, pages, page_ld, (uint4*)out);
  return spark_launch_rc(__func__);
}

extern "C" int spark_latent_rows(const void* q_full, const void* cache, const int* pos, const int* rows, const int* row_slot,
                                 const int* pages, int page_ld, int n, int H, int Lp, int Rp, float scale, const void* gate, int ldg,
                                 const float* sink, void* out, int f32, cudaStream_t s) {
  if (n <= 0) return 0;
  if (Lp > 1024 || H > 65535 || ((Lp + Rp) & 3)) return -5;
  SPARK_BY_TYPE(f32, spark_launch_pdl(latent_rows_kernel<T>, dim3(n, H), dim3(128), (Lp + Rp + 128) * 4, s, dim3(1, 1, 1),
                                      (const T*)q_full, (const T*)cache, pos, rows, row_slot, pages, page_ld, H, Lp, Rp, scale,
                                      (const T*)gate, ldg, sink, (T*)out))
  return spark_launch_rc(__func__);
}

// bf16.  gate (optional): at column 0 of its rows, one logit per head or (gate_all) one per output column.  -6: the shape does not fit shared memory (the caller uses spark_latent_rows).
extern "C" int spark_latent_prefill(const void* q, int ldq, const void* kv, int ldkv, const void* lat, int ldlat, const int* segs,
                                    int nseg, int max_rows, int H, int Dp, int Rp, int V, int Vp, int Lp, float scale,
                                    const void* gate, int ldg, int gate_all, const float* sink, void* out, int ldo, cudaStream_t s) {
  if (nseg <= 0) return 0;
  if ((gate_all && (reinterpret_cast<uintptr_t>(gate) & 3)) || (reinterpret_cast<uintptr_t>(out) & 3)) return -5;
  if ((Dp | Rp | Vp | Lp) & 15 || Vp < V || (ldq | ldkv | ldlat) & 7) return -5;
  LatentPrefill a;
  a.q = (const __nv_bfloat16*)q; a.kv = (const __nv_bfloat16*)kv; a.lat = (const __nv_bfloat16*)lat; a.gate = (const __nv_bfloat16*)gate;
  a.out = (__nv_bfloat16*)out; a.segs = segs; a.ldq = ldq; a.ldkv = ldkv; a.ldlat = ldlat; a.ldg = ldg; a.ldo = ldo;
  a.H = H; a.Dp = Dp; a.Rp = Rp; a.V = V; a.Vp = Vp; a.Lp = Lp; a.scale_log2 = scale * 1.4426950408889634f;
  a.sink = sink; a.gate_all = gate_all;
  if (Vp <= 32) return launch_latent_prefill<32, 8>(a, nseg, max_rows, s);
  if (Vp <= 64) return launch_latent_prefill<64, 8>(a, nseg, max_rows, s);
  if (Vp <= 128) return launch_latent_prefill<128, 8>(a, nseg, max_rows, s);
  if (Vp <= 256) return launch_latent_prefill<256, 8>(a, nseg, max_rows, s);
  return -6;
}
