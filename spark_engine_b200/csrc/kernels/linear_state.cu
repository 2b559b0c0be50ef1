// Linear recurrences without a delta rule, one kernel family for three mechanisms.  Per head, with state S [D, V] (fp32):
//
//   scalar decay (MODE 0):  S_t = a S_{t-1} + k_t v_t^T,          o_t = S_t^T q_t       (a: one constant per head)
//   channel decay (MODE 1): o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T
//                           (w_t in (0, 1) per key channel and token, u a bonus of the current token)
//   channel decay (MODE 2): S_t = diag(w_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t
//
// Outputs are multiplied by a constant `qscale`.
//
// linear_seq_kernel   rows one after the other, state in registers: decode and verify rows, short portions, and the whole
//                     32-bit mode.  `commit` = 0 leaves the state untouched; a later launch with the accepted row counts
//                     replays and commits.
// chunked form        64-row chunks on tensor cores for prompts (bf16 activations):
//   linear_chunk_u      U_c = sum_j exp(G_C - G_j) k_j v_j^T of every chunk, all chunks in parallel
//   linear_scan         S <- exp(G_C) S + U_c over the chunks of a segment, element by element; leaves the state ENTERING each
//                       chunk in place of U_c and the final state in the slot
//   linear_chunk_o      o = (q exp(E)) S_in + sum_{j < i} (sum_c q_ic k_jc exp(E_ic - G_jc)) v_j + diagonal term
// G is the running log decay inside the chunk (inclusive), E_i = G_i in MODES 0 and 2, G_{i-1} in MODE 1.  Exponents are
// only ever taken of differences that are <= 0 (for a pair of 16-row blocks the reference point lies between them, the
// diagonal blocks are summed pair by pair), so no decay is too strong for fp32.  bf16 enters as operands that are bf16
// anyway (activations of the projections); every fp32 factor (state, weights, decayed keys) goes to the tensor cores as
// a two-term bf16 sum, accumulated in fp32.
#include "../common/rows.cuh"

namespace spark {

struct LinearArgs {
  const void *q, *k, *v;         // T: row r, head h, channel d at [r * ld + h * hs + d]
  int ldq, ldk, ldv, hsk, hsv;
  const float* log2a;            // MODE 0: log2 of the decay [H]
  const float* logw;             // MODES 1, 2: natural log of the decay [R, H * D]
  const float* u;                // MODE 1: [H, D]
  float* S;                      // [slots, H, D, V]
  const int* seg;                // [nseg][4]: slot, first row, rows, first position
  const int* n_rows;             // optional per segment: rows to process (commit of accepted rows)
  float* o;                      // [R, H * V]
  const float* h32; float* carried; int width;   // MODE 1: rows the token shift reads, and the per-slot carried row
  int H, D, V, commit, act;      // act: SiLU on q, k, v
  float qscale;
};

// Channel decays formed by the sequential kernel itself: ln(sigmoid(w2 z + b)) / tau; z, w2 in the activation type, rank % 8 == 0.
struct LowRankDecay {
  const void *z, *w2;
  const float* b;
  int ldz, ldw, rank;
  float inv_tau;
};

// ------------------------------------------------------------------------------------------------ sequential form
// grid (ceil(V / 32), H, nseg); 2 * DP threads: lane = value column, warp = 16 key channels
template <typename T, int DP, int MODE>
__global__ void __launch_bounds__(2 * DP)
linear_seq_kernel(const __grid_constant__ LinearArgs a, const __grid_constant__ LowRankDecay lr) {
  constexpr int NP = DP / 16;
  __shared__ float sq[2][DP], sk[2][DP], sw[MODE ? 2 : 1][DP], su[DP], red[2][NP][32];
  pdl_wait();
  const int h = blockIdx.y, sg = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int slot = a.seg[sg * 4], r0 = a.seg[sg * 4 + 1];
  int n = a.seg[sg * 4 + 2];
  if (a.n_rows != nullptr) n = min(n, a.n_rows[sg]);
  if (n <= 0) return;
  const int D = a.D, V = a.V, vcol = blockIdx.x * 32 + lane;
  const bool vin = vcol < V;
  const T* q = static_cast<const T*>(a.q) + h * a.hsk;
  const T* k = static_cast<const T*>(a.k) + h * a.hsk;
  const T* v = static_cast<const T*>(a.v) + h * a.hsv;
  float s[16];
  float* Sp = a.S + ((static_cast<size_t>(slot) * a.H + h) * D + warp * 16) * V + vcol;
#pragma unroll
  for (int j = 0; j < 16; ++j) s[j] = (vin && warp * 16 + j < D) ? Sp[static_cast<size_t>(j) * V] : 0.f;
  float lam = 0.f;
  if (MODE == 0) lam = exp2f(a.log2a[h]);
  if (MODE == 1 && tid < DP) su[tid] = tid < D ? a.u[h * D + tid] : 0.f;
  // thread tid < DP stages q and w of channel tid, the others k
  const int c = tid < DP ? tid : tid - DP;
  auto fetch = [&](int t, float& x, float& w, float& vv) {
    const size_t r = r0 + t;
    x = c < D ? (tid < DP ? ldf(q + r * a.ldq + c) : ldf(k + r * a.ldk + c)) : 0.f;
    w = 0.f;
    if (MODE >= 1 && tid < DP && c < D) {
      if (MODE == 2 && lr.z != nullptr) {
        const T* z = static_cast<const T*>(lr.z) + r * lr.ldz;
        const T* w2 = static_cast<const T*>(lr.w2) + static_cast<size_t>(h * D + c) * lr.ldw;
        float e = lr.b[h * D + c];
        for (int i = 0; i < lr.rank; i += 8) {
          const float4 z0 = ldf4(z + i), z1 = ldf4(z + i + 4), w0 = ldf4(w2 + i), w1 = ldf4(w2 + i + 4);
          e = fmaf(z0.x, w0.x, e); e = fmaf(z0.y, w0.y, e); e = fmaf(z0.z, w0.z, e); e = fmaf(z0.w, w0.w, e);
          e = fmaf(z1.x, w1.x, e); e = fmaf(z1.y, w1.y, e); e = fmaf(z1.z, w1.z, e); e = fmaf(z1.w, w1.w, e);
        }
        w = log_sigmoid_decay(e, lr.inv_tau);
      } else {
        w = a.logw[r * (static_cast<size_t>(a.H) * D) + h * D + c];
      }
    }
    vv = vin ? ldf(v + r * a.ldv + vcol) : 0.f;
  };
  float x, w, vv;
  fetch(0, x, w, vv);
  for (int t = 0; t < n; ++t) {
    const int b = t & 1;
    if (a.act) { x = silu_f(x); vv = silu_f(vv); }
    if (tid < DP) { sq[b][c] = x; if (MODE >= 1) sw[b][c] = c < D ? expf(w) : 0.f; }
    else sk[b][c] = x;
    const float val = vv;
    if (t + 1 < n) fetch(t + 1, x, w, vv);
    __syncthreads();
    if (t > 0 && warp == (t - 1) % NP && vin) {               // partial sums of the previous row
      float o = 0.f;
#pragma unroll
      for (int p = 0; p < NP; ++p) o += red[b ^ 1][p][lane];
      a.o[(static_cast<size_t>(r0) + t - 1) * (static_cast<size_t>(a.H) * V) + h * V + vcol] = o * a.qscale;
    }
    float o = 0.f;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const int d = warp * 16 + j;
      const float kv = sk[b][d] * val;
      if (MODE == 0) {
        s[j] = fmaf(lam, s[j], kv);
        o = fmaf(sq[b][d], s[j], o);
      } else if (MODE == 2) {
        s[j] = fmaf(sw[b][d], s[j], kv);
        o = fmaf(sq[b][d], s[j], o);
      } else {
        o = fmaf(sq[b][d], fmaf(su[d], kv, s[j]), o);
        s[j] = fmaf(sw[b][d], s[j], kv);
      }
    }
    red[b][warp][lane] = o;
  }
  __syncthreads();
  if (warp == 0 && vin) {
    float o = 0.f;
#pragma unroll
    for (int p = 0; p < NP; ++p) o += red[(n - 1) & 1][p][lane];
    a.o[(static_cast<size_t>(r0) + n - 1) * (static_cast<size_t>(a.H) * V) + h * V + vcol] = o * a.qscale;
  }
  if (a.commit) {
#pragma unroll
    for (int j = 0; j < 16; ++j)
      if (vin && warp * 16 + j < D) Sp[static_cast<size_t>(j) * V] = s[j];
    if (MODE == 1 && a.h32 != nullptr && blockIdx.x == 0 && h == 0)
      for (int i = tid; i < a.width; i += 2 * DP)
        a.carried[static_cast<size_t>(slot) * a.width + i] = a.h32[(static_cast<size_t>(r0) + n - 1) * a.width + i];
  }
}

// ------------------------------------------------------------------------------------------------ chunked form
constexpr int LC = 64;             // rows per chunk
constexpr int LVT = 64;            // value columns per tile
constexpr int LVS = LVT + 8;       // smem row stride of a value tile

__device__ __forceinline__ void lc_ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lc_ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x, y as two-term bf16 sums, packed for an MMA fragment
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
// 2^x on the special-function unit (relative error about 2^-22; 0 for very negative x)
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float LOG2E = 1.4426950408889634f;
__device__ __forceinline__ void split1(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(x);
  lo = __float2bfloat16(x - __bfloat162float(hi));
}

// Row tile [LC][lds] of one head by 128 threads: rows past nv and channels past ncol are zero; SiLU optional.  Whole aligned
// tiles are fetched as a batch of 16-byte loads.  dst rows are 4-byte aligned.
__device__ __forceinline__ void put_rows8(__nv_bfloat16* dst, const float (&f)[8], int act) {
#pragma unroll
  for (int e = 0; e < 8; e += 2) {
    const float x = act ? silu_t<__nv_bfloat16>(f[e]) : f[e], y = act ? silu_t<__nv_bfloat16>(f[e + 1]) : f[e + 1];
    *reinterpret_cast<__nv_bfloat162*>(dst + e) = __floats2bfloat162_rn(x, y);
  }
}
template <int COLS>
__device__ __forceinline__ void load_rows(__nv_bfloat16* __restrict__ dst, int lds, const __nv_bfloat16* __restrict__ src, int ld,
                                          int nv, int ncol, int act) {
  constexpr int PER = LC * (COLS / 8) / 128;                 // 16-byte pieces per thread
  const bool whole = nv == LC && ncol >= COLS && (ld & 7) == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0;
  if (whole) {
    uint4 u[PER];
#pragma unroll
    for (int b = 0; b < PER; ++b) {
      const int i = threadIdx.x + b * 128, r = i / (COLS / 8), c = (i % (COLS / 8)) * 8;
      u[b] = *reinterpret_cast<const uint4*>(src + static_cast<size_t>(r) * ld + c);
    }
#pragma unroll
    for (int b = 0; b < PER; ++b) {
      const int i = threadIdx.x + b * 128, r = i / (COLS / 8), c = (i % (COLS / 8)) * 8;
      const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&u[b]);
      float f[8];
#pragma unroll
      for (int e = 0; e < 4; ++e) { const float2 t = __bfloat1622float2(p[e]); f[2 * e] = t.x; f[2 * e + 1] = t.y; }
      put_rows8(dst + r * lds + c, f, act);
    }
    return;
  }
  for (int i = threadIdx.x; i < LC * (COLS / 8); i += 128) {
    const int r = i / (COLS / 8), c = (i % (COLS / 8)) * 8;
    float f[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = (r < nv && c + e < ncol) ? __bfloat162float(src[static_cast<size_t>(r) * ld + c + e]) : 0.f;
    put_rows8(dst + r * lds + c, f, act);
  }
}
// Log decays [LC][ldg] (base 2) of one head: zero past nv / ncol.
template <int COLS>
__device__ __forceinline__ void load_decays(float* __restrict__ G, int ldg, const float* __restrict__ lw, size_t ld, int nv, int ncol) {
  constexpr int PER = LC * (COLS / 4) / 128;
  if (nv == LC && ncol >= COLS && (ld & 3) == 0 && (reinterpret_cast<uintptr_t>(lw) & 15) == 0) {
    float4 u[PER];
#pragma unroll
    for (int b = 0; b < PER; ++b) {
      const int i = threadIdx.x + b * 128;
      u[b] = ldf4(lw + (i / (COLS / 4)) * ld + (i % (COLS / 4)) * 4);
    }
#pragma unroll
    for (int b = 0; b < PER; ++b) {
      const int i = threadIdx.x + b * 128;
      float2* d = reinterpret_cast<float2*>(G + (i / (COLS / 4)) * ldg + (i % (COLS / 4)) * 4);
      d[0] = make_float2(LOG2E * u[b].x, LOG2E * u[b].y);
      d[1] = make_float2(LOG2E * u[b].z, LOG2E * u[b].w);
    }
    return;
  }
  for (int i = threadIdx.x; i < LC * COLS; i += 128) {
    const int r = i / COLS, c = i % COLS;
    G[r * ldg + c] = (r < nv && c < ncol) ? LOG2E * lw[r * ld + c] : 0.f;
  }
}

// grid (chunks, H, ceil(V / 64)); 128 threads.  ws_u [chunk][H][D][V]; MODES 1, 2 also ws_d [chunk][H][D] = exp(G_C).
template <int DP, int MODE>
__global__ void __launch_bounds__(128)
linear_chunk_u_kernel(const __grid_constant__ LinearArgs a, const int* __restrict__ chunks, float* __restrict__ ws_u,
                      float* __restrict__ ws_d) {
  constexpr int LDK = DP + 8;
  extern __shared__ __align__(16) uint8_t smem_lu[];
  __nv_bfloat16* Kh = reinterpret_cast<__nv_bfloat16*>(smem_lu);       // [64][LDK] decayed keys, high / low part
  __nv_bfloat16* Kl = Kh + LC * LDK;
  __nv_bfloat16* Vs = Kl + LC * LDK;                                     // [64][LVS]
  const int ci = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * LVT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int sg = chunks[2 * ci], t0 = chunks[2 * ci + 1] * LC;
  const int n = a.seg[sg * 4 + 2], nv = min(LC, n - t0);
  const size_t r0 = static_cast<size_t>(a.seg[sg * 4 + 1]) + t0;
  const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(a.k) + r0 * a.ldk + h * a.hsk;
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.v) + r0 * a.ldv + h * a.hsv + v0;
  load_rows<LVT>(Vs, LVS, v, a.ldv, nv, a.V - v0, a.act);
  if (MODE == 0) {
    load_rows<DP>(Kh, LDK, k, a.ldk, nv, a.D, a.act);
    __syncthreads();
    const float l2 = a.log2a[h];
    for (int i = tid; i < LC * (DP / 2); i += 128) {
      const int r = i / (DP / 2), c = (i - r * (DP / 2)) * 2;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Kh + r * LDK + c));
      const int e = nv - 1 - r;
      const float w = e > 0 ? exp2f(l2 * e) : (e == 0 ? 1.f : 0.f);
      uint32_t hi, lo;
      split2(x.x * w, x.y * w, hi, lo);
      *reinterpret_cast<uint32_t*>(Kh + r * LDK + c) = hi;
      *reinterpret_cast<uint32_t*>(Kl + r * LDK + c) = lo;
    }
  } else {
    float* G = reinterpret_cast<float*>(smem_lu + (2 * LC * LDK + LC * LVS) * 2);     // [64][DP] running sums, base 2
    float* gsum = G + LC * DP;                                                         // [16][DP] of four-row groups
    load_rows<DP>(Kh, LDK, k, a.ldk, nv, a.D, 0);
    load_decays<DP>(G, DP, a.logw + r0 * (static_cast<size_t>(a.H) * a.D) + h * a.D, static_cast<size_t>(a.H) * a.D, nv, a.D);
    __syncthreads();
    for (int i = tid; i < 16 * DP; i += 128) {                            // four rows at a time, then the 16 group sums
      const int gr = i / DP, c = i - gr * DP;
      float s = 0.f;
#pragma unroll
      for (int r = 0; r < 4; ++r) { s += G[(gr * 4 + r) * DP + c]; G[(gr * 4 + r) * DP + c] = s; }
      gsum[i] = s;
    }
    __syncthreads();
    for (int c = tid; c < DP; c += 128) {
      float s = 0.f;
#pragma unroll
      for (int gr = 0; gr < 16; ++gr) { const float x = gsum[gr * DP + c]; gsum[gr * DP + c] = s; s += x; }
      gsum[16 * DP + c] = s;
      if (c < a.D && v0 == 0) ws_d[(static_cast<size_t>(ci) * a.H + h) * a.D + c] = ex2(s);
    }
    __syncthreads();
    for (int i = tid; i < LC * (DP / 2); i += 128) {
      const int r = i / (DP / 2), c = (i - r * (DP / 2)) * 2;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Kh + r * LDK + c));
      const float w0 = ex2(gsum[16 * DP + c] - (G[r * DP + c] + gsum[(r >> 2) * DP + c]));
      const float w1 = ex2(gsum[16 * DP + c + 1] - (G[r * DP + c + 1] + gsum[(r >> 2) * DP + c + 1]));
      uint32_t hi, lo;
      split2(x.x * w0, x.y * w1, hi, lo);
      *reinterpret_cast<uint32_t*>(Kh + r * LDK + c) = hi;
      *reinterpret_cast<uint32_t*>(Kl + r * LDK + c) = lo;
    }
  }
  __syncthreads();
  const int g = lane >> 2, t = lane & 3;
  float* U = ws_u + (static_cast<size_t>(ci) * a.H + h) * a.D * a.V + v0;
  for (int mt = warp; mt < DP / 16; mt += 4) {
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) { acc[i][0] = 0.f; acc[i][1] = 0.f; acc[i][2] = 0.f; acc[i][3] = 0.f; }
#pragma unroll
    for (int ks = 0; ks < LC / 16; ++ks) {
      // A = K^T: rows = channels, contraction over tokens; transposed 8x8 loads of [token][channel]
      uint32_t ah[4], al[4];
      const int off = (ks * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + mt * 16 + ((lane >> 3) & 1) * 8;
      lc_ldsm4t(ah, Kh + off);
      lc_ldsm4t(al, Kl + off);
#pragma unroll
      for (int np = 0; np < LVT / 16; ++np) {
        uint32_t b[4];
        lc_ldsm4t(b, Vs + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LVS + np * 16 + (lane >> 4) * 8);
        lc_mma(acc[2 * np], ah, b[0], b[1]); lc_mma(acc[2 * np + 1], ah, b[2], b[3]);
        lc_mma(acc[2 * np], al, b[0], b[1]); lc_mma(acc[2 * np + 1], al, b[2], b[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int d = mt * 16 + g + (e >> 1) * 8, vv = i * 8 + 2 * t;
        float* p = U + static_cast<size_t>(d) * a.V + vv;
        if (d < a.D && v0 + vv + 1 < a.V && (a.V & 1) == 0) *reinterpret_cast<float2*>(p) = make_float2(acc[i][e], acc[i][e + 1]);
        else if (d < a.D) {
          if (v0 + vv < a.V) p[0] = acc[i][e];
          if (v0 + vv + 1 < a.V) p[1] = acc[i][e + 1];
        }
      }
  }
}

// grid (ceil(D * V / (128 VEC)), H, nseg); 128 threads: VEC consecutive state elements each (V % VEC == 0).
template <int MODE, int VEC>
__global__ void __launch_bounds__(128)
linear_scan_kernel(const __grid_constant__ LinearArgs a, const int* __restrict__ seg_chunk0, float* __restrict__ ws_u,
                   const float* __restrict__ ws_d) {
  const int h = blockIdx.y, sg = blockIdx.z, e = (blockIdx.x * 128 + threadIdx.x) * VEC;
  const int DV = a.D * a.V;
  const int slot = a.seg[sg * 4], r0 = a.seg[sg * 4 + 1], n = a.seg[sg * 4 + 2];
  const int nch = (n + LC - 1) / LC;
  if (e < DV) {
    struct Vec { float v[VEC]; };
    auto ld = [](const float* p) {
      Vec x;
      if (VEC == 4) { const float4 t = ldf4(p); x.v[0] = t.x; x.v[VEC > 1 ? 1 : 0] = t.y; x.v[VEC > 2 ? 2 : 0] = t.z; x.v[VEC > 3 ? 3 : 0] = t.w; }
      if (VEC == 1) x.v[0] = *p;
      return x;
    };
    auto st = [](float* p, const Vec& x) {
      if (VEC == 4) stf4(p, make_float4(x.v[0], x.v[VEC > 1 ? 1 : 0], x.v[VEC > 2 ? 2 : 0], x.v[VEC > 3 ? 3 : 0]));
      else *p = x.v[0];
    };
    float* Sp = a.S + (static_cast<size_t>(slot) * a.H + h) * DV + e;
    Vec s = ld(Sp);
    const size_t cst = static_cast<size_t>(a.H) * DV;
    float* u = ws_u + (static_cast<size_t>(seg_chunk0[sg]) * a.H + h) * DV + e;
    const float* dd = MODE ? ws_d + (static_cast<size_t>(seg_chunk0[sg]) * a.H + h) * a.D + e / a.V : nullptr;
    const float full = MODE ? 0.f : exp2f(a.log2a[h] * LC);
    const float last = MODE ? 0.f : exp2f(a.log2a[h] * (n - (nch - 1) * LC));
    constexpr int PF = 8;                                      // chunks of loads in flight: batch c0 + 8 is fetched while c0 is scanned
    Vec x[PF], nx[PF];
    float dc[PF], nd[PF];
    auto fetch = [&](int c0, Vec (&xx)[PF], float (&dx)[PF]) {
#pragma unroll
      for (int i = 0; i < PF; ++i) {
        const int c = min(c0 + i, nch - 1);
        xx[i] = ld(u + c * cst);
        dx[i] = MODE ? dd[static_cast<size_t>(c) * a.H * a.D] : (c == nch - 1 ? last : full);
      }
    };
    fetch(0, x, dc);
    for (int c0 = 0; c0 < nch; c0 += PF) {
      if (c0 + PF < nch) fetch(c0 + PF, nx, nd);
#pragma unroll
      for (int i = 0; i < PF; ++i) {
        if (c0 + i < nch) {
          st(u + (c0 + i) * cst, s);
#pragma unroll
          for (int k = 0; k < VEC; ++k) s.v[k] = fmaf(dc[i], s.v[k], x[i].v[k]);
        }
        x[i] = nx[i]; dc[i] = nd[i];
      }
    }
    if (a.commit) st(Sp, s);
  }
  if (MODE == 1 && a.commit && a.h32 != nullptr && blockIdx.x == 0 && h == 0)
    for (int i = threadIdx.x; i < a.width; i += 128)
      a.carried[static_cast<size_t>(slot) * a.width + i] = a.h32[(static_cast<size_t>(r0) + n - 1) * a.width + i];
}

template <int DP, int MODE>
struct ChunkOSmem {
  static constexpr int LDK = DP + 8, LDR = DP + 2, LDG = DP + 2;      // pairs of channels, rows spread over the banks
  static constexpr int KHL = MODE ? 2 * LC * LDK * 2 : 2 * LC * LDK * 2;            // MODE 0: Q | K;  MODE 1: K^ high | low
  static constexpr int RAW = MODE ? 2 * LC * LDR * 2 : 0;                             // MODE 1: r, k as they are
  static constexpr int G = MODE ? ((LC * LDG * 4 + 15) / 16 * 16) : 0;
  static constexpr int DG = MODE ? 4 * 16 * 17 * 4 : 0;
  static constexpr int VB = LC * LVS * 2, SB = 2 * DP * LVS * 2;
  static constexpr int TOTAL = KHL + RAW + G + DG + VB + SB;
};

// grid (chunks, H, ceil(V / 64)); 128 threads: warp w owns rows 16w .. 16w + 15 of the chunk.
template <int DP, int MODE>
__global__ void __launch_bounds__(128)
linear_chunk_o_kernel(const __grid_constant__ LinearArgs a, const int* __restrict__ chunks, const float* __restrict__ ws_u) {
  using SM = ChunkOSmem<DP, MODE>;
  constexpr int LDK = SM::LDK, LDR = SM::LDR, LDG = SM::LDG;
  extern __shared__ __align__(16) uint8_t smem_lo[];
  __nv_bfloat16* A0 = reinterpret_cast<__nv_bfloat16*>(smem_lo);        // MODE 0: Q;  MODE 1: K^ high
  __nv_bfloat16* A1 = A0 + LC * LDK;                                     // MODE 0: K;  MODE 1: K^ low
  __nv_bfloat16* Rr = reinterpret_cast<__nv_bfloat16*>(smem_lo + SM::KHL);
  __nv_bfloat16* Kr = Rr + LC * LDR;
  float* G = reinterpret_cast<float*>(smem_lo + SM::KHL + SM::RAW);      // inclusive running log decay, base 2
  float* Dg = reinterpret_cast<float*>(smem_lo + SM::KHL + SM::RAW + SM::G);   // diagonal 16 x 16 blocks
  __nv_bfloat16* Vs = reinterpret_cast<__nv_bfloat16*>(smem_lo + SM::KHL + SM::RAW + SM::G + SM::DG);
  __nv_bfloat16* Sh = Vs + LC * LVS;                                     // [DP][LVS] state entering the chunk, high / low
  __nv_bfloat16* Sl = Sh + DP * LVS;
  const int ci = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * LVT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int sg = chunks[2 * ci], t0 = chunks[2 * ci + 1] * LC;
  const int n = a.seg[sg * 4 + 2], nv = min(LC, n - t0);
  const size_t r0 = static_cast<size_t>(a.seg[sg * 4 + 1]) + t0;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + r0 * a.ldq + h * a.hsk;
  const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(a.k) + r0 * a.ldk + h * a.hsk;
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.v) + r0 * a.ldv + h * a.hsv;
  const float l2 = MODE == 0 ? a.log2a[h] : 0.f;
  const int row_lo = warp * 16 + g, row_hi = row_lo + 8;
  // the state that entered the chunk (this CTA's value columns) as two-term sums
  const float* Sin = ws_u + (static_cast<size_t>(ci) * a.H + h) * a.D * a.V;
  auto load_state = [&]() {
    auto put = [&](int d, int c, float4 x) {
      uint32_t h0, l0, h1, l1;
      split2(x.x, x.y, h0, l0);
      split2(x.z, x.w, h1, l1);
      *reinterpret_cast<uint2*>(Sh + d * LVS + c) = make_uint2(h0, h1);
      *reinterpret_cast<uint2*>(Sl + d * LVS + c) = make_uint2(l0, l1);
    };
    constexpr int PER = DP * (LVT / 4) / 128, BT = PER < 8 ? PER : 8;
    if (a.D == DP && v0 + LVT <= a.V && (a.V & 3) == 0) {
      for (int b0 = 0; b0 < PER; b0 += BT) {
        float4 x[BT];
#pragma unroll
        for (int b = 0; b < BT; ++b) {
          const int i = tid + (b0 + b) * 128;
          x[b] = ldf4(Sin + static_cast<size_t>(i / (LVT / 4)) * a.V + v0 + (i % (LVT / 4)) * 4);
        }
#pragma unroll
        for (int b = 0; b < BT; ++b) { const int i = tid + (b0 + b) * 128; put(i / (LVT / 4), (i % (LVT / 4)) * 4, x[b]); }
      }
      return;
    }
    for (int i = tid; i < DP * (LVT / 4); i += 128) {
      const int d = i / (LVT / 4), c = (i % (LVT / 4)) * 4;
      const float* p = Sin + static_cast<size_t>(d) * a.V + v0 + c;
      float f[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) f[e] = (d < a.D && v0 + c + e < a.V) ? p[e] : 0.f;
      put(d, c, make_float4(f[0], f[1], f[2], f[3]));
    }
  };
  if (MODE == 0) {
    load_rows<DP>(A0, LDK, q, a.ldq, nv, a.D, a.act);
    load_rows<DP>(A1, LDK, k, a.ldk, nv, a.D, a.act);
    load_state();
    load_rows<LVT>(Vs, LVS, v + v0, a.ldv, nv, a.V - v0, a.act);
    __syncthreads();
  } else {
    load_state();
    load_rows<LVT>(Vs, LVS, v + v0, a.ldv, nv, a.V - v0, a.act);
    load_rows<DP>(Rr, LDR, q, a.ldq, nv, a.D, 0);
    load_rows<DP>(Kr, LDR, k, a.ldk, nv, a.D, 0);
    load_decays<DP>(G, LDG, a.logw + r0 * (static_cast<size_t>(a.H) * a.D) + h * a.D, static_cast<size_t>(a.H) * a.D, nv, a.D);
    __syncthreads();
    for (int i = tid; i < 4 * DP; i += 128) {                              // running sums of the 16-row blocks, then across them
      const int b = i / DP, c = i % DP;
      float s = 0.f;
#pragma unroll
      for (int r = 0; r < 16; ++r) { s += G[(b * 16 + r) * LDG + c]; G[(b * 16 + r) * LDG + c] = s; }
    }
    __syncthreads();
    for (int i = tid; i < 3 * DP; i += 128) {
      const int b = 1 + i / DP, c = i % DP;
      float add = 0.f;
      for (int p = 0; p < b; ++p) add += G[(p * 16 + 15) * LDG + c];
      Dg[i] = add;                                                           // (scratch until the diagonal blocks are formed)
    }
    __syncthreads();
    for (int i = tid; i < 48 * DP; i += 128) { const int r = 16 + i / DP, c = i % DP; G[r * LDG + c] += Dg[(r / 16 - 1) * DP + c]; }
    __syncthreads();
    // keys decayed to the end of their own 16-row block
    for (int i = tid; i < LC * (DP / 2); i += 128) {
      const int r = i / (DP / 2), c = (i - r * (DP / 2)) * 2;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Kr + r * LDR + c));
      const float2 e = *reinterpret_cast<const float2*>(G + (r | 15) * LDG + c), f = *reinterpret_cast<const float2*>(G + r * LDG + c);
      uint32_t hi, lo;
      split2(x.x * ex2(e.x - f.x), x.y * ex2(e.y - f.y), hi, lo);
      *reinterpret_cast<uint32_t*>(A0 + r * LDK + c) = hi;
      *reinterpret_cast<uint32_t*>(A1 + r * LDK + c) = lo;
    }
    // diagonal blocks, pair by pair: i > j decayed from j to i - 1 (MODE 2: to i), i == j weighted by the bonus
    for (int p = lane; p < 136; p += 32) {
      int i = 0;
      while ((i + 1) * (i + 2) / 2 <= p) ++i;
      const int j = p - i * (i + 1) / 2;
      const int ri = warp * 16 + i, rj = warp * 16 + j;
      float s = 0.f;
      if (i == j) {
        for (int c = 0; c < a.D; ++c)
          s = fmaf(__bfloat162float(Rr[ri * LDR + c]) * (MODE == 1 ? a.u[h * a.D + c] : 1.f), __bfloat162float(Kr[rj * LDR + c]), s);
      } else {
        float s1 = 0.f;
#pragma unroll 4
        for (int c = 0; c < DP; c += 2) {                                  // (channels past D are zero)
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Rr + ri * LDR + c));
          const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Kr + rj * LDR + c));
          const float2 e = *reinterpret_cast<const float2*>(G + (MODE == 1 ? ri - 1 : ri) * LDG + c), f = *reinterpret_cast<const float2*>(G + rj * LDG + c);
          s = fmaf(x.x * y.x, ex2(e.x - f.x), s);
          s1 = fmaf(x.y * y.y, ex2(e.y - f.y), s1);
        }
        s += s1;
      }
      Dg[(warp * 16 + i) * 17 + j] = s;
    }
    __syncthreads();
  }
  // receptance fragment of one 16-channel step: r exp(E - ref), E = G of the previous row (MODE 2: of the row)
  auto rfrag = [&](int ks, int ref_row, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = (e & 1) ? row_hi : row_lo, c = ks * 16 + 2 * t + (e >> 1) * 8;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Rr + row * LDR + c));
      const int er = MODE == 1 ? row - 1 : row;
      const float2 E = er >= 0 ? *reinterpret_cast<const float2*>(G + er * LDG + c) : make_float2(0.f, 0.f);
      const float2 f = ref_row >= 0 ? *reinterpret_cast<const float2*>(G + ref_row * LDG + c) : make_float2(0.f, 0.f);
      split2(x.x * ex2(E.x - f.x), x.y * ex2(E.y - f.y), hi[e], lo[e]);
    }
  };
  // ---- weights of the keys of this chunk as MMA operands: two-term sums, key blocks 0 .. warp
  uint32_t ph[4][4], pl[4][4];
#pragma unroll
  for (int kb = 0; kb < 4; ++kb) {
#pragma unroll
    for (int e = 0; e < 4; ++e) { ph[kb][e] = 0u; pl[kb][e] = 0u; }
    if (kb > warp) continue;
    float s[2][4] = {};
    if (MODE == 0) {
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t x[4], b[4];
        lc_ldsm4(x, A0 + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + ks * 16 + (lane >> 4) * 8);
        lc_ldsm4(b, A1 + (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
        lc_mma(s[0], x, b[0], b[1]); lc_mma(s[1], x, b[2], b[3]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = ((e >> 1) ? row_hi : row_lo) - (kb * 16 + i * 8 + 2 * t + (e & 1));
          s[i][e] = d > 0 ? s[i][e] * exp2f(l2 * d) : (d == 0 ? s[i][e] : 0.f);
        }
    } else if (kb < warp) {
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t xh[4], xl[4], bh[4], bl[4];
        rfrag(ks, kb * 16 + 15, xh, xl);
        const int off = (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + ks * 16 + ((lane >> 3) & 1) * 8;
        lc_ldsm4(bh, A0 + off);
        lc_ldsm4(bl, A1 + off);
        lc_mma(s[0], xh, bh[0], bh[1]); lc_mma(s[1], xh, bh[2], bh[3]);
        lc_mma(s[0], xh, bl[0], bl[1]); lc_mma(s[1], xh, bl[2], bl[3]);
        lc_mma(s[0], xl, bh[0], bh[1]); lc_mma(s[1], xl, bh[2], bh[3]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int ri = g + (e >> 1) * 8, cj = i * 8 + 2 * t + (e & 1);
          s[i][e] = cj <= ri ? Dg[(warp * 16 + ri) * 17 + cj] : 0.f;
        }
    }
    split2(s[0][0], s[0][1], ph[kb][0], pl[kb][0]); split2(s[0][2], s[0][3], ph[kb][1], pl[kb][1]);
    split2(s[1][0], s[1][1], ph[kb][2], pl[kb][2]); split2(s[1][2], s[1][3], ph[kb][3], pl[kb][3]);
  }
  const float dec_lo = MODE == 0 ? exp2f(l2 * (row_lo + 1)) : 1.f, dec_hi = MODE == 0 ? exp2f(l2 * (row_hi + 1)) : 1.f;
  {
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    // the state that entered the chunk
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks) {
      uint32_t xh[4], xl[4];
      if (MODE == 0) lc_ldsm4(xh, A0 + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + ks * 16 + (lane >> 4) * 8);
      else rfrag(ks, -1, xh, xl);
#pragma unroll
      for (int np = 0; np < LVT / 16; ++np) {
        uint32_t bh[4], bl[4];
        const int off = (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LVS + np * 16 + (lane >> 4) * 8;
        lc_ldsm4t(bh, Sh + off);
        lc_ldsm4t(bl, Sl + off);
        lc_mma(o[2 * np], xh, bh[0], bh[1]); lc_mma(o[2 * np + 1], xh, bh[2], bh[3]);
        lc_mma(o[2 * np], xh, bl[0], bl[1]); lc_mma(o[2 * np + 1], xh, bl[2], bl[3]);
        if (MODE >= 1) { lc_mma(o[2 * np], xl, bh[0], bh[1]); lc_mma(o[2 * np + 1], xl, bh[2], bh[3]); }
      }
    }
    if (MODE == 0) {
#pragma unroll
      for (int i = 0; i < 8; ++i) { o[i][0] *= dec_lo; o[i][1] *= dec_lo; o[i][2] *= dec_hi; o[i][3] *= dec_hi; }
    }
    // the keys of the chunk
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      if (kb > warp) continue;
#pragma unroll
      for (int np = 0; np < LVT / 16; ++np) {
        uint32_t b[4];
        lc_ldsm4t(b, Vs + (kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LVS + np * 16 + (lane >> 4) * 8);
        lc_mma(o[2 * np], ph[kb], b[0], b[1]); lc_mma(o[2 * np + 1], ph[kb], b[2], b[3]);
        lc_mma(o[2 * np], pl[kb], b[0], b[1]); lc_mma(o[2 * np + 1], pl[kb], b[2], b[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int row = e ? row_hi : row_lo, c = v0 + i * 8 + 2 * t;
        float* p = a.o + (r0 + row) * (static_cast<size_t>(a.H) * a.V) + h * a.V + c;
        const float x = o[i][e] * a.qscale, y = o[i][e + 1] * a.qscale;
        if (row < nv && c + 1 < a.V && (a.V & 1) == 0) *reinterpret_cast<float2*>(p) = make_float2(x, y);
        else if (row < nv) {
          if (c < a.V) p[0] = x;
          if (c + 1 < a.V) p[1] = y;
        }
      }
  }
}

template <int DP, int MODE>
static int launch_chunked(const LinearArgs& a, const int* chunks, int n_chunks, const int* chunk0, int nseg, float* ws_u, float* ws_d,
                          cudaStream_t s) {
  auto ku = linear_chunk_u_kernel<DP, MODE>;
  auto ko = linear_chunk_o_kernel<DP, MODE>;
  constexpr int SU = (2 * LC * (DP + 8) + LC * LVS) * 2 + (MODE ? (LC + 17) * DP * 4 : 0), SO = ChunkOSmem<DP, MODE>::TOTAL;
  static bool done = false;
  if (!done) {
    cudaFuncSetAttribute(ku, cudaFuncAttributeMaxDynamicSharedMemorySize, SU);
    cudaFuncSetAttribute(ko, cudaFuncAttributeMaxDynamicSharedMemorySize, SO);
    done = true;
  }
  ku<<<dim3(n_chunks, a.H, (a.V + LVT - 1) / LVT), 128, SU, s>>>(a, chunks, ws_u, ws_d);
  if (a.V % 4 == 0) linear_scan_kernel<MODE, 4><<<dim3((a.D * a.V + 511) / 512, a.H, nseg), 128, 0, s>>>(a, chunk0, ws_u, ws_d);
  else linear_scan_kernel<MODE, 1><<<dim3((a.D * a.V + 127) / 128, a.H, nseg), 128, 0, s>>>(a, chunk0, ws_u, ws_d);
  ko<<<dim3(n_chunks, a.H, (a.V + LVT - 1) / LVT), 128, SO, s>>>(a, chunks, ws_u);
  return spark_launch_rc("spark_linear_chunked");
}

template <typename T, int MODE>
static int launch_seq(const LinearArgs& a, int nseg, cudaStream_t s, const LowRankDecay& lr = LowRankDecay{}) {
  const dim3 grid((a.V + 31) / 32, a.H, nseg);
#define SPARK_LSEQ(DP) spark_launch_pdl(linear_seq_kernel<T, DP, MODE>, grid, dim3(2 * DP), 0, s, dim3(1, 1, 1), a, lr)
  if (a.D <= 32) SPARK_LSEQ(32);
  else if (a.D <= 64) SPARK_LSEQ(64);
  else if (a.D <= 128) SPARK_LSEQ(128);
  else if (a.D <= 256) SPARK_LSEQ(256);
  else if (a.D <= 512) SPARK_LSEQ(512);
  else return -5;
#undef SPARK_LSEQ
  return spark_launch_rc("spark_linear_seq");
}

static LinearArgs linear_args(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, int hsk, int hsv,
                              const float* log2a, const float* logw, const float* u, float* S, const int* seg, const int* n_rows,
                              float* o, const float* h32, float* carried, int width, int H, int D, int V, int commit, int act,
                              float qscale) {
  LinearArgs a;
  a.q = q; a.k = k; a.v = v; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.hsk = hsk; a.hsv = hsv;
  a.log2a = log2a; a.logw = logw; a.u = u; a.S = S; a.seg = seg; a.n_rows = n_rows; a.o = o;
  a.h32 = h32; a.carried = carried; a.width = width; a.H = H; a.D = D; a.V = V; a.commit = commit; a.act = act; a.qscale = qscale;
  return a;
}

}  // namespace spark

using namespace spark;

#define SPARK_LINEAR_PARAMS                                                                                              \
  const void *q, int ldq, const void *k, int ldk, const void *v, int ldv, int hsk, int hsv, const float *log2a,          \
      const float *logw, const float *u, float *S, const int *seg, const int *n_rows, float *o, const float *h32,        \
      float *carried, int width, int H, int D, int V, int commit, int act, float qscale
#define SPARK_LINEAR_ARGS \
  linear_args(q, ldq, k, ldk, v, ldv, hsk, hsv, log2a, logw, u, S, seg, n_rows, o, h32, carried, width, H, D, V, commit, act, qscale)

// log2a != nullptr: scalar decay per head; else channel decay (logw), with a bonus u or (u null) without.
extern "C" int spark_linear_seq(SPARK_LINEAR_PARAMS, int nseg, int f32, cudaStream_t s) {
  if (nseg <= 0) return 0;
  const LinearArgs a = SPARK_LINEAR_ARGS;
  if (log2a) return f32 ? launch_seq<float, 0>(a, nseg, s) : launch_seq<__nv_bfloat16, 0>(a, nseg, s);
  if (u) return f32 ? launch_seq<float, 1>(a, nseg, s) : launch_seq<__nv_bfloat16, 1>(a, nseg, s);
  return f32 ? launch_seq<float, 2>(a, nseg, s) : launch_seq<__nv_bfloat16, 2>(a, nseg, s);
}

// Channel decay without a bonus, the decays from their low-rank rows.
extern "C" int spark_linear_seq_lowrank(SPARK_LINEAR_PARAMS, int nseg, const LowRankDecay* lr, int f32, cudaStream_t s) {
  if (nseg <= 0) return 0;
  if (log2a || u || lr->rank <= 0 || ((lr->rank | lr->ldz | lr->ldw) & 7) || !(lr->inv_tau > 0.f) ||
      ((reinterpret_cast<uintptr_t>(lr->z) | reinterpret_cast<uintptr_t>(lr->w2)) & 15)) return -5;
  const LinearArgs a = SPARK_LINEAR_ARGS;
  return f32 ? launch_seq<float, 2>(a, nseg, s, *lr) : launch_seq<__nv_bfloat16, 2>(a, nseg, s, *lr);
}

// chunks: int [n_chunks][2] = (segment, chunk in segment); chunk0: int [nseg] first chunk of a segment.  D <= 128.
// ws_u: fp32 [n_chunks, H, D, V]; ws_d: fp32 [n_chunks, H, D] (channel decay).
extern "C" int spark_linear_chunked(SPARK_LINEAR_PARAMS, int nseg, const int* chunks, int n_chunks, const int* chunk0, float* ws_u,
                                    float* ws_d, cudaStream_t s) {
  if (nseg <= 0 || n_chunks <= 0) return 0;
  if (n_rows != nullptr || D > 128) return -5;
  const LinearArgs a = SPARK_LINEAR_ARGS;
#define SPARK_LCH(DP) (log2a ? launch_chunked<DP, 0>(a, chunks, n_chunks, chunk0, nseg, ws_u, ws_d, s) \
         : u  ? launch_chunked<DP, 1>(a, chunks, n_chunks, chunk0, nseg, ws_u, ws_d, s) \
                             : launch_chunked<DP, 2>(a, chunks, n_chunks, chunk0, nseg, ws_u, ws_d, s))
  if (D <= 32) return SPARK_LCH(32);
  if (D <= 64) return SPARK_LCH(64);
  return SPARK_LCH(128);
#undef SPARK_LCH
}
