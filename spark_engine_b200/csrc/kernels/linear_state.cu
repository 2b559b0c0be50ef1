// Linear recurrences without a delta rule, one kernel family for two mechanisms.  Per head, with state S [D, V] (fp32):
//
//   scalar decay (MODE 0):  S_t = a S_{t-1} + k_t v_t^T,          o_t = S_t^T q_t       (a: one constant per head)
//   channel decay (MODE 1): o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T
//                           (w_t in (0, 1) per key channel and token, u a bonus of the current token)
//
// linear_seq_kernel   rows one after the other, state in registers: decode and verify rows, short portions, and the whole
//                     32-bit mode.  `commit` = 0 leaves the state untouched; a later launch with the accepted row counts
//                     replays and commits.
// chunked form        64-row chunks on tensor cores for prompts (bf16 activations):
//   linear_chunk_u      U_c = sum_j exp(G_C - G_j) k_j v_j^T of every chunk, all chunks in parallel
//   linear_scan         S <- exp(G_C) S + U_c over the chunks of a segment, element by element; leaves the state ENTERING each
//                       chunk in place of U_c and the final state in the slot
//   linear_chunk_o      o = (q exp(E)) S_in + sum_{j < i} (sum_c q_ic k_jc exp(E_ic - G_jc)) v_j + diagonal term
// G is the running log decay inside the chunk (inclusive), E_i = G_i in MODE 0 and G_{i-1} in MODE 1.  Exponents are
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
  const float* logw;             // MODE 1: natural log of the decay [R, H * D]
  const float* u;                // MODE 1: [H, D]
  float* S;                      // [slots, H, D, V]
  const int* seg;                // [nseg][4]: slot, first row, rows, first position
  const int* n_rows;             // optional per segment: rows to process (commit of accepted rows)
  float* o;                      // [R, H * V]
  const float* h32; float* carried; int width;   // MODE 1: rows the token shift reads, and the per-slot carried row
  int H, D, V, commit, act;      // act: SiLU on q, k, v
};

// ------------------------------------------------------------------------------------------------ sequential form
// grid (ceil(V / 32), H, nseg); 2 * DP threads: lane = value column, warp = 16 key channels
template <typename T, int DP, int MODE>
__global__ void __launch_bounds__(2 * DP)
linear_seq_kernel(const __grid_constant__ LinearArgs a) {
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
    w = (MODE == 1 && tid < DP && c < D) ? a.logw[r * (static_cast<size_t>(a.H) * D) + h * D + c] : 0.f;
    vv = vin ? ldf(v + r * a.ldv + vcol) : 0.f;
  };
  float x, w, vv;
  fetch(0, x, w, vv);
  for (int t = 0; t < n; ++t) {
    const int b = t & 1;
    if (a.act) { x = silu_f(x); vv = silu_f(vv); }
    if (tid < DP) { sq[b][c] = x; if (MODE == 1) sw[b][c] = c < D ? expf(w) : 0.f; }
    else sk[b][c] = x;
    const float val = vv;
    if (t + 1 < n) fetch(t + 1, x, w, vv);
    __syncthreads();
    if (t > 0 && warp == (t - 1) % NP && vin) {               // partial sums of the previous row
      float o = 0.f;
#pragma unroll
      for (int p = 0; p < NP; ++p) o += red[b ^ 1][p][lane];
      a.o[(static_cast<size_t>(r0) + t - 1) * (static_cast<size_t>(a.H) * V) + h * V + vcol] = o;
    }
    float o = 0.f;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const int d = warp * 16 + j;
      const float kv = sk[b][d] * val;
      if (MODE == 0) {
        s[j] = fmaf(lam, s[j], kv);
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
    a.o[(static_cast<size_t>(r0) + n - 1) * (static_cast<size_t>(a.H) * V) + h * V + vcol] = o;
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
__device__ __forceinline__ void split1(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(x);
  lo = __float2bfloat16(x - __bfloat162float(hi));
}

// Row tile [LC][ld] of one head: rows past nv and channels past D are zero; SiLU optional.
template <int COLS>
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, int lds, const __nv_bfloat16* src, int ld, int nv, int ncol, int act) {
  for (int i = threadIdx.x; i < LC * (COLS / 8); i += blockDim.x) {
    const int r = i / (COLS / 8), c = (i - r * (COLS / 8)) * 8;
    float f[8];
    const __nv_bfloat16* p = src + static_cast<size_t>(r) * ld + c;
    if (r < nv && c + 8 <= ncol && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
      const uint4 u = *reinterpret_cast<const uint4*>(p);
      const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
      for (int e = 0; e < 4; ++e) { const float2 t = __bfloat1622float2(b[e]); f[2 * e] = t.x; f[2 * e + 1] = t.y; }
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = (r < nv && c + e < ncol) ? __bfloat162float(p[e]) : 0.f;
    }
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const float x = act ? silu_f(f[e]) : f[e], y = act ? silu_f(f[e + 1]) : f[e + 1];
      *reinterpret_cast<__nv_bfloat162*>(dst + r * lds + c + e) = __floats2bfloat162_rn(x, y);
    }
  }
}

// grid (chunks, H, ceil(V / 64)); 128 threads.  ws_u [chunk][H][D][V]; MODE 1 also ws_d [chunk][H][D] = exp(G_C).
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
    const float l2 = a.log2a[h];
    for (int i = tid; i < LC * DP; i += 128) {
      const int r = i / DP, c = i - r * DP;
      float x = (r < nv && c < a.D) ? __bfloat162float(k[static_cast<size_t>(r) * a.ldk + c]) : 0.f;
      if (a.act) x = __bfloat162float(__float2bfloat16(silu_f(x)));
      const int e = nv - 1 - r;
      x = e > 0 ? x * exp2f(l2 * e) : (e == 0 ? x : 0.f);
      split1(x, Kh[r * LDK + c], Kl[r * LDK + c]);
    }
  } else {
    for (int c = tid; c < DP; c += 128) {                                 // suffix sums: G_C - G_j, last row first
      float g = 0.f;
      const float* lw = a.logw + r0 * (static_cast<size_t>(a.H) * a.D) + h * a.D + c;
#pragma unroll 8
      for (int r = LC - 1; r >= 0; --r) {
        float x = 0.f;
        if (r < nv && c < a.D) {
          x = __bfloat162float(k[static_cast<size_t>(r) * a.ldk + c]) * expf(g);
          g += lw[static_cast<size_t>(r) * a.H * a.D];
        }
        split1(x, Kh[r * LDK + c], Kl[r * LDK + c]);
      }
      if (c < a.D && v0 == 0) ws_d[(static_cast<size_t>(ci) * a.H + h) * a.D + c] = expf(g);
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
      for (int e = 0; e < 4; ++e) {
        const int d = mt * 16 + g + (e >> 1) * 8, vv = i * 8 + 2 * t + (e & 1);
        if (d < a.D && v0 + vv < a.V) U[static_cast<size_t>(d) * a.V + vv] = acc[i][e];
      }
  }
}

// grid (ceil(D * V / 256), H, nseg); 256 threads: one state element each.
template <int MODE>
__global__ void __launch_bounds__(256)
linear_scan_kernel(const __grid_constant__ LinearArgs a, const int* __restrict__ seg_chunk0, float* __restrict__ ws_u,
                   const float* __restrict__ ws_d) {
  const int h = blockIdx.y, sg = blockIdx.z, e = blockIdx.x * 256 + threadIdx.x;
  const int DV = a.D * a.V;
  const int slot = a.seg[sg * 4], r0 = a.seg[sg * 4 + 1], n = a.seg[sg * 4 + 2];
  const int nch = (n + LC - 1) / LC;
  if (e < DV) {
    float* Sp = a.S + (static_cast<size_t>(slot) * a.H + h) * DV + e;
    float s = *Sp;
    const size_t cst = static_cast<size_t>(a.H) * DV;
    float* u = ws_u + (static_cast<size_t>(seg_chunk0[sg]) * a.H + h) * DV + e;
    const float* dd = MODE ? ws_d + (static_cast<size_t>(seg_chunk0[sg]) * a.H + h) * a.D + e / a.V : nullptr;
    const float full = MODE ? 0.f : exp2f(a.log2a[h] * LC);
    const float last = MODE ? 0.f : exp2f(a.log2a[h] * (n - (nch - 1) * LC));
    for (int c0 = 0; c0 < nch; c0 += 8) {                      // eight chunks of loads in flight
      float x[8], dc[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int c = c0 + i;
        x[i] = c < nch ? u[c * cst] : 0.f;
        dc[i] = MODE ? (c < nch ? dd[static_cast<size_t>(c) * a.H * a.D] : 0.f) : (c == nch - 1 ? last : full);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (c0 + i < nch) { u[(c0 + i) * cst] = s; s = fmaf(dc[i], s, x[i]); }
      }
    }
    if (a.commit) *Sp = s;
  }
  if (MODE == 1 && a.commit && a.h32 != nullptr && blockIdx.x == 0 && h == 0)
    for (int i = threadIdx.x; i < a.width; i += 256)
      a.carried[static_cast<size_t>(slot) * a.width + i] = a.h32[(static_cast<size_t>(r0) + n - 1) * a.width + i];
}

template <int DP, int MODE>
struct ChunkOSmem {
  static constexpr int LDK = DP + 8, LDR = DP + 2, LDG = DP + 1;
  static constexpr int KHL = MODE ? 2 * LC * LDK * 2 : 2 * LC * LDK * 2;            // MODE 0: Q | K;  MODE 1: K^ high | low
  static constexpr int RAW = MODE ? 2 * LC * LDR * 2 : 0;                             // MODE 1: r, k as they are
  static constexpr int G = MODE ? ((LC * LDG * 4 + 15) / 16 * 16) : 0;
  static constexpr int DG = MODE ? 4 * 16 * 17 * 4 : 0;
  static constexpr int VB = LC * LVS * 2, SB = 2 * DP * LVS * 2;
  static constexpr int TOTAL = KHL + RAW + G + DG + VB + SB;
};

// grid (chunks, H); 128 threads: warp w owns rows 16w .. 16w + 15 of the chunk.
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
  float* G = reinterpret_cast<float*>(smem_lo + SM::KHL + SM::RAW);      // inclusive running log decay
  float* Dg = reinterpret_cast<float*>(smem_lo + SM::KHL + SM::RAW + SM::G);   // diagonal 16 x 16 blocks
  __nv_bfloat16* Vs = reinterpret_cast<__nv_bfloat16*>(smem_lo + SM::KHL + SM::RAW + SM::G + SM::DG);
  __nv_bfloat16* Sh = Vs + LC * LVS;                                     // [DP][LVS] state entering the chunk, high / low
  __nv_bfloat16* Sl = Sh + DP * LVS;
  const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int sg = chunks[2 * ci], t0 = chunks[2 * ci + 1] * LC;
  const int n = a.seg[sg * 4 + 2], nv = min(LC, n - t0);
  const size_t r0 = static_cast<size_t>(a.seg[sg * 4 + 1]) + t0;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + r0 * a.ldq + h * a.hsk;
  const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(a.k) + r0 * a.ldk + h * a.hsk;
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.v) + r0 * a.ldv + h * a.hsv;
  const float l2 = MODE == 0 ? a.log2a[h] : 0.f;
  const int row_lo = warp * 16 + g, row_hi = row_lo + 8;
  if (MODE == 0) {
    load_rows<DP>(A0, LDK, q, a.ldq, nv, a.D, a.act);
    load_rows<DP>(A1, LDK, k, a.ldk, nv, a.D, a.act);
    __syncthreads();
  } else {
    for (int i = tid; i < LC * DP; i += 128) {
      const int r = i / DP, c = i - r * DP;
      const bool in = r < nv && c < a.D;
      Rr[r * LDR + c] = in ? q[static_cast<size_t>(r) * a.ldq + c] : __float2bfloat16(0.f);
      Kr[r * LDR + c] = in ? k[static_cast<size_t>(r) * a.ldk + c] : __float2bfloat16(0.f);
      G[r * LDG + c] = in ? a.logw[(r0 + r) * (static_cast<size_t>(a.H) * a.D) + h * a.D + c] : 0.f;
    }
    __syncthreads();
    for (int c = tid; c < DP; c += 128) {
      float s = 0.f;
#pragma unroll 8
      for (int r = 0; r < LC; ++r) { s += G[r * LDG + c]; G[r * LDG + c] = s; }
    }
    __syncthreads();
    // keys decayed to the end of their own 16-row block
    for (int i = tid; i < LC * DP; i += 128) {
      const int r = i / DP, c = i - r * DP;
      split1(__bfloat162float(Kr[r * LDR + c]) * expf(G[(r | 15) * LDG + c] - G[r * LDG + c]), A0[r * LDK + c], A1[r * LDK + c]);
    }
    // diagonal blocks, pair by pair: i > j decayed from j to i - 1, i == j weighted by the bonus
    for (int p = lane; p < 136; p += 32) {
      int i = 0;
      while ((i + 1) * (i + 2) / 2 <= p) ++i;
      const int j = p - i * (i + 1) / 2;
      const int ri = warp * 16 + i, rj = warp * 16 + j;
      float s = 0.f;
      if (i == j) {
        for (int c = 0; c < a.D; ++c)
          s = fmaf(__bfloat162float(Rr[ri * LDR + c]) * a.u[h * a.D + c], __bfloat162float(Kr[rj * LDR + c]), s);
      } else {
        for (int c = 0; c < a.D; ++c)
          s = fmaf(__bfloat162float(Rr[ri * LDR + c]) * __bfloat162float(Kr[rj * LDR + c]),
                   expf(G[(ri - 1) * LDG + c] - G[rj * LDG + c]), s);
      }
      Dg[(warp * 16 + i) * 17 + j] = s;
    }
    __syncthreads();
  }
  // receptance fragment of one 16-channel step: r exp(E - ref), E = G of the previous row
  auto rfrag = [&](int ks, int ref_row, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = (e & 1) ? row_hi : row_lo, c = ks * 16 + 2 * t + (e >> 1) * 8;
      float x[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float E = row > 0 ? G[(row - 1) * LDG + c + i] : 0.f;
        const float ref = ref_row >= 0 ? G[ref_row * LDG + c + i] : 0.f;
        x[i] = __bfloat162float(Rr[row * LDR + c + i]) * expf(E - ref);
      }
      split2(x[0], x[1], hi[e], lo[e]);
    }
  };
  // ---- weights of the keys of this chunk as MMA operands: two-term sums, key blocks 0 .. warp
  uint32_t ph[4][4], pl[4][4];
  const float p_lo_rows = 0.f; (void)p_lo_rows;
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
  const float* Sin = ws_u + (static_cast<size_t>(ci) * a.H + h) * a.D * a.V;
  for (int v0 = 0; v0 < a.V; v0 += LVT) {
    if (v0) __syncthreads();
    load_rows<LVT>(Vs, LVS, v + v0, a.ldv, nv, a.V - v0, a.act);
    for (int i = tid; i < DP * LVT; i += 128) {
      const int d = i / LVT, c = i - d * LVT;
      split1((d < a.D && v0 + c < a.V) ? Sin[static_cast<size_t>(d) * a.V + v0 + c] : 0.f, Sh[d * LVS + c], Sl[d * LVS + c]);
    }
    __syncthreads();
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
        if (MODE == 1) { lc_mma(o[2 * np], xl, bh[0], bh[1]); lc_mma(o[2 * np + 1], xl, bh[2], bh[3]); }
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
      for (int e = 0; e < 4; ++e) {
        const int row = (e >> 1) ? row_hi : row_lo, c = v0 + i * 8 + 2 * t + (e & 1);
        if (row < nv && c < a.V) a.o[(r0 + row) * (static_cast<size_t>(a.H) * a.V) + h * a.V + c] = o[i][e];
      }
  }
}

template <int DP, int MODE>
static int launch_chunked(const LinearArgs& a, const int* chunks, int n_chunks, const int* chunk0, int nseg, float* ws_u, float* ws_d,
                          cudaStream_t s) {
  auto ku = linear_chunk_u_kernel<DP, MODE>;
  auto ko = linear_chunk_o_kernel<DP, MODE>;
  constexpr int SU = (2 * LC * (DP + 8) + LC * LVS) * 2, SO = ChunkOSmem<DP, MODE>::TOTAL;
  static bool done = false;
  if (!done) {
    cudaFuncSetAttribute(ku, cudaFuncAttributeMaxDynamicSharedMemorySize, SU);
    cudaFuncSetAttribute(ko, cudaFuncAttributeMaxDynamicSharedMemorySize, SO);
    done = true;
  }
  ku<<<dim3(n_chunks, a.H, (a.V + LVT - 1) / LVT), 128, SU, s>>>(a, chunks, ws_u, ws_d);
  linear_scan_kernel<MODE><<<dim3((a.D * a.V + 255) / 256, a.H, nseg), 256, 0, s>>>(a, chunk0, ws_u, ws_d);
  ko<<<dim3(n_chunks, a.H), 128, SO, s>>>(a, chunks, ws_u);
  return spark_launch_rc("spark_linear_chunked");
}

template <typename T, int MODE>
static int launch_seq(const LinearArgs& a, int nseg, cudaStream_t s) {
  const dim3 grid((a.V + 31) / 32, a.H, nseg);
#define SPARK_LSEQ(DP) spark_launch_pdl(linear_seq_kernel<T, DP, MODE>, grid, dim3(2 * DP), 0, s, dim3(1, 1, 1), a)
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
                              float* o, const float* h32, float* carried, int width, int H, int D, int V, int commit, int act) {
  LinearArgs a;
  a.q = q; a.k = k; a.v = v; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.hsk = hsk; a.hsv = hsv;
  a.log2a = log2a; a.logw = logw; a.u = u; a.S = S; a.seg = seg; a.n_rows = n_rows; a.o = o;
  a.h32 = h32; a.carried = carried; a.width = width; a.H = H; a.D = D; a.V = V; a.commit = commit; a.act = act;
  return a;
}

}  // namespace spark

using namespace spark;

#define SPARK_LINEAR_PARAMS                                                                                              \
  const void *q, int ldq, const void *k, int ldk, const void *v, int ldv, int hsk, int hsv, const float *log2a,          \
      const float *logw, const float *u, float *S, const int *seg, const int *n_rows, float *o, const float *h32,        \
      float *carried, int width, int H, int D, int V, int commit, int act
#define SPARK_LINEAR_ARGS \
  linear_args(q, ldq, k, ldk, v, ldv, hsk, hsv, log2a, logw, u, S, seg, n_rows, o, h32, carried, width, H, D, V, commit, act)

// log2a != nullptr: scalar decay per head; else channel decay (logw, u).
extern "C" int spark_linear_seq(SPARK_LINEAR_PARAMS, int nseg, int f32, cudaStream_t s) {
  if (nseg <= 0) return 0;
  const LinearArgs a = SPARK_LINEAR_ARGS;
  if (log2a) return f32 ? launch_seq<float, 0>(a, nseg, s) : launch_seq<__nv_bfloat16, 0>(a, nseg, s);
  return f32 ? launch_seq<float, 1>(a, nseg, s) : launch_seq<__nv_bfloat16, 1>(a, nseg, s);
}

// chunks: int [n_chunks][2] = (segment, chunk in segment); chunk0: int [nseg] first chunk of a segment.  D <= 128.
// ws_u: fp32 [n_chunks, H, D, V]; ws_d: fp32 [n_chunks, H, D] (channel decay).
extern "C" int spark_linear_chunked(SPARK_LINEAR_PARAMS, int nseg, const int* chunks, int n_chunks, const int* chunk0, float* ws_u,
                                    float* ws_d, cudaStream_t s) {
  if (nseg <= 0 || n_chunks <= 0) return 0;
  if (n_rows != nullptr || D > 128) return -5;
  const LinearArgs a = SPARK_LINEAR_ARGS;
#define SPARK_LCH(DP) (log2a ? launch_chunked<DP, 0>(a, chunks, n_chunks, chunk0, nseg, ws_u, ws_d, s) \
                             : launch_chunked<DP, 1>(a, chunks, n_chunks, chunk0, nseg, ws_u, ws_d, s))
  if (D <= 32) return SPARK_LCH(32);
  if (D <= 64) return SPARK_LCH(64);
  return SPARK_LCH(128);
#undef SPARK_LCH
}
