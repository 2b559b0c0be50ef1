// Residual updates over tiles of consecutive rows of a sequence, for blocks whose sublayers read
//
//   h + conv(h),  h = RMS norm of the new residual over groups of channels,  conv a causal convolution over time with a few taps
//                 per channel (the sequence's last taps - 1 rows h are its state)
//
// and whose residual may become a learned sum of all earlier layer results ("depth average").  One launch does all of it:
//
//   row_tiles     x = res + update; depth average: stack[k] = x, x = sum_j a[j] stack[j]; res_out = x; h; out = h + conv(h)
//   tail_advance  the state behind rows that were verified and accepted
//
// A CTA owns a tile of rows and walks them in order; every thread keeps its channels' last taps - 1 values of h in shared memory,
// so the convolution costs no further pass over the rows.  The rows just before a tile are recomputed (`res` is left as it is; the
// results go to `res_out`), the first tile of a segment starts from the slot's state and writes the state behind the segment.
// A row's bits do not depend on how the sequence was cut.  Norms, sums, state and convolution are fp32.
#include "../common/row_update.cuh"

namespace spark {

struct RowTiles {
  RowUpdate u;                 // no norm of the update, no layer norm
  float* res_out;              // [R, H]
  float* stack;                // [k + 1 or more][R, H] (null: no depth average)
  const float* avg;            // [k + 1]
  const float* conv_w;         // [taps, H]
  float* tail;                 // [slots, taps - 1, H]
  float* rows;                 // [R, H]: h, for a pass whose state advances later (commit 0)
  const int* segs;             // [n][4]: slot, first row, rows, first position (null: one segment of R rows)
  int k, groups, taps, tile, commit, R;      // taps 0: no convolution
};

template <int N> struct Ch { float v[N]; };
template <int N> __device__ __forceinline__ Ch<N> ldc(const float* p) {
  Ch<N> c;
  if constexpr (N == 4) { const float4 f = ldf4(p); c.v[0] = f.x; c.v[1] = f.y; c.v[2] = f.z; c.v[3] = f.w; }
  else c.v[0] = *p;
  return c;
}
template <int N> __device__ __forceinline__ Ch<N> ldc(const __nv_bfloat16* p) {
  Ch<N> c;
  if constexpr (N == 4) { const float4 f = ldf4(p); c.v[0] = f.x; c.v[1] = f.y; c.v[2] = f.z; c.v[3] = f.w; }
  else c.v[0] = ldf(p);
  return c;
}
template <int N, typename T> __device__ __forceinline__ void stc(T* p, const Ch<N>& c) {
  if constexpr (N == 4) stf4(p, make_float4(c.v[0], c.v[1], c.v[2], c.v[3]));
  else stf(p, c.v[0]);
}

// grid (tiles, segments); whole warps, N channels per thread and step.  WIDE: groups are multiples of a warp's 128 channels.
// Shared memory: [taps - 1][H] ring | [H] row | WIDE: [2][H / 128] partial sums, [H / 128] first piece of a piece's group; else
// [H / N] squares and [groups] factors.
template <typename T, int N, bool WIDE>
__global__ void __launch_bounds__(1024)
row_tiles_kernel(const __grid_constant__ RowTiles a) {
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  if (gridDim.x * gridDim.y <= 148) pdl_trigger();           // decode rounds: the successor's CTAs find room beside these
  const int H = a.u.H, t = threadIdx.x, nt = blockDim.x, lane = t & 31, warp = t >> 5, past = a.taps > 1 ? a.taps - 1 : 0;
  const int* sg = a.segs ? a.segs + blockIdx.y * 4 : nullptr;
  const int slot = sg ? sg[0] : 0, r0 = sg ? sg[1] : 0, n = sg ? sg[2] : a.R;
  const int j0 = blockIdx.x * a.tile, jn = min(n, j0 + a.tile);
  if (j0 >= n) return;
  float* ring = sm;
  float* xs = ring + static_cast<size_t>(past) * H;
  float* red = xs + H;
  int* first = reinterpret_cast<int*>(red + 2 * (H >> 7));    // WIDE
  if (WIDE) {
    const int per = (H / a.groups) >> 7;
    for (int c = t; c < H >> 7; c += nt) first[c] = c / per * per;      // (read behind the first row's barrier)
  }
  const size_t plane = static_cast<size_t>(a.R) * H;
  const int gs = H / a.groups;
  const float inv_gs = 1.f / gs;
  const bool has = a.u.delta != nullptr || a.u.y != nullptr;
  const float one = a.u.one_plus ? 1.f : 0.f;
  T* out = static_cast<T*>(a.u.out);
  int turn = 0;

  // the row's new residual, channels i ..; `own`: this CTA stores it
  auto assemble = [&](int r, int i, bool own) {
    const size_t at = static_cast<size_t>(r) * H + i;
    Ch<N> x = ldc<N>(a.u.res + at);
    if (has) {
      Ch<N> u{};
      if (a.u.delta) u = ldc<N>(a.u.delta + at);
      else {
        for (int s0 = 0; s0 < a.u.slots; s0 += 4) {           // four slots' rows in flight, added in slot order
          Ch<N> p[4]; float w[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int pi = r * a.u.slots + s0 + q;
            const bool live = s0 + q < a.u.slots && a.u.ids[pi] >= 0;
            w[q] = live ? (a.u.wts ? a.u.wts[pi] : 1.f) : 0.f;
            p[q] = Ch<N>{};
            if (live) p[q] = ldc<N>(a.u.y + static_cast<size_t>(a.u.inv ? a.u.inv[pi] : pi) * H + i);
          }
#pragma unroll
          for (int q = 0; q < 4; ++q)
#pragma unroll
            for (int e = 0; e < N; ++e) u.v[e] = fmaf(w[q], p[q].v[e], u.v[e]);
        }
        const float self = a.u.self_w ? a.u.self_w[r] : 0.f;
        if (self != 0.f) {
          const Ch<N> p = ldc<N>(static_cast<const T*>(a.u.self_x) + at);
#pragma unroll
          for (int e = 0; e < N; ++e) u.v[e] = fmaf(self, p.v[e], u.v[e]);
        }
        if (a.u.shared) {
          const float g = a.u.sg ? a.u.sg[r] : 1.f;
          const Ch<N> p = ldc<N>(a.u.shared + at);
#pragma unroll
          for (int e = 0; e < N; ++e) u.v[e] = fmaf(g, p.v[e], u.v[e]);
        }
      }
      if (a.u.scale) {
        const Ch<N> m = ldc<N>(a.u.scale + i);
#pragma unroll
        for (int e = 0; e < N; ++e) u.v[e] *= m.v[e];
      }
#pragma unroll
      for (int e = 0; e < N; ++e) x.v[e] += u.v[e];
    }
    if (a.stack) {
      if (own) stc<N>(a.stack + a.k * plane + at, x);
      Ch<N> y{};
      for (int k0 = 0; k0 < a.k; k0 += 4) {                   // four results in flight, added in layer order
        Ch<N> p[4]; float w[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const bool live = k0 + q < a.k;
          w[q] = live ? a.avg[k0 + q] : 0.f;
          p[q] = Ch<N>{};
          if (live) p[q] = ldc<N>(a.stack + (k0 + q) * plane + at);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
          for (int e = 0; e < N; ++e) y.v[e] = fmaf(w[q], p[q].v[e], y.v[e]);
      }
      const float w = a.avg[a.k];
#pragma unroll
      for (int e = 0; e < N; ++e) x.v[e] = fmaf(w, x.v[e], y.v[e]);
    }
    if (own && a.res_out) stc<N>(a.res_out + at, x);
    return x;
  };

  // row j of the segment: use(i, h) for the thread's channels
  auto row = [&](int j, bool own, auto&& use) {
    const int r = r0 + j;
    float* part = red + (WIDE ? (turn & 1) * (H >> 7) : 0);
    ++turn;
    for (int i = t * N; i < H; i += nt * N) {
      const Ch<N> x = assemble(r, i, own);
      stc<N>(xs + i, x);
      if (a.u.norm) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < N; ++e) ss = fmaf(x.v[e], x.v[e], ss);
        if (WIDE) {
          ss = warp_sum(ss);
          if (lane == 0) part[i >> 7] = ss;
        } else part[i / N] = ss;
      }
    }
    float* fac = red + H / N;
    if (a.u.norm) {
      __syncthreads();
      if (!WIDE) {                                            // a warp per group
        for (int g = warp; g < a.groups; g += nt >> 5) {
          float s = 0.f;
          for (int c = lane; c < gs / N; c += 32) s += part[g * (gs / N) + c];
          s = warp_sum(s);
          if (lane == 0) fac[g] = rsqrtf(s * inv_gs + a.u.eps);
        }
        __syncthreads();
      }
    }
    for (int i = t * N; i < H; i += nt * N) {
      Ch<N> h = ldc<N>(xs + i);
      if (a.u.norm) {
        float rs;
        if (WIDE) {                                           // a warp's channels are of one group
          const int c0 = first[i >> 7];
          float s = 0.f;
          for (int c = lane; c < gs >> 7; c += 32) s += part[c0 + c];
          rs = rsqrtf(warp_sum(s) * inv_gs + a.u.eps);
        } else rs = fac[i / gs];
        const Ch<N> w = ldc<N>(a.u.w + i);
#pragma unroll
        for (int e = 0; e < N; ++e) h.v[e] = h.v[e] * rs * (one + w.v[e]);
      }
      use(i, h);
    }
  };

  int q = past;                                               // ring entry of row j: (j - first walked row) % past
  int j = j0;
  if (past > 0) {
    if (j0 == 0) {
      for (int i = t * N; i < H; i += nt * N)
        for (int p = 0; p < past; ++p) stc<N>(ring + p * H + i, ldc<N>(a.tail + (static_cast<size_t>(slot) * past + p) * H + i));
    } else {
      j = j0 - past;                                          // (tile >= taps - 1: these rows belong to the tile before)
      for (int p = 0; p < past; ++p, ++j) row(j, false, [&](int i, const Ch<N>& h) { stc<N>(ring + p * H + i, h); });
    }
    q = 0;
  }
  for (; j < jn; ++j) {
    const size_t base = static_cast<size_t>(r0 + j) * H;
    row(j, true, [&](int i, const Ch<N>& h) {
      Ch<N> y = h;
      if (a.taps > 0) {
        int e0 = q;                                           // the oldest entry
        for (int p = 0; p < past; ++p) {
          const Ch<N> w = ldc<N>(a.conv_w + p * H + i), b = ldc<N>(ring + e0 * H + i);
#pragma unroll
          for (int e = 0; e < N; ++e) y.v[e] = fmaf(w.v[e], b.v[e], y.v[e]);
          if (++e0 == past) e0 = 0;
        }
        const Ch<N> w = ldc<N>(a.conv_w + past * H + i);
#pragma unroll
        for (int e = 0; e < N; ++e) y.v[e] = fmaf(w.v[e], h.v[e], y.v[e]);
        if (past > 0) stc<N>(ring + q * H + i, h);
        if (a.rows) stc<N>(a.rows + base + i, h);
      }
      if (out) stc<N>(out + base + i, y);
      if (a.u.out32) stc<N>(a.u.out32 + base + i, y);
    });
    if (past > 0 && ++q == past) q = 0;
  }
  if (past == 0 || !a.commit || j0 != 0) return;
  float* tail = a.tail + static_cast<size_t>(slot) * past * H;
  if (jn == n) {                                              // the ring holds the last rows, entry q the oldest
    for (int i = t * N; i < H; i += nt * N)
      for (int p = 0, e0 = q; p < past; ++p) {
        stc<N>(tail + p * H + i, ldc<N>(ring + e0 * H + i));
        if (++e0 == past) e0 = 0;
      }
  } else {
    for (int p = 0; p < past; ++p) row(n - past + p, false, [&](int i, const Ch<N>& h) { stc<N>(tail + p * H + i, h); });
  }
}

// grid (ceil(H / 256), segments); 256 threads: a channel each.
__global__ void __launch_bounds__(256)
tail_advance_kernel(float* __restrict__ tail, const float* __restrict__ rows, const int* __restrict__ segs, const int* __restrict__ n_rows,
                    int past, int H) {
  pdl_wait();
  const int i = blockIdx.x * 256 + threadIdx.x;
  const int* sg = segs + blockIdx.y * 4;
  const int n = n_rows ? min(max(n_rows[blockIdx.y], 0), sg[2]) : sg[2];
  if (i >= H || n == 0) return;
  float* s = tail + static_cast<size_t>(sg[0]) * past * H + i;
  for (int p = 0; p < past; ++p) {                            // ascending: an entry is read before a later row replaces it
    const int j = n - past + p;
    s[p * H] = j >= 0 ? rows[static_cast<size_t>(sg[1] + j) * H + i] : s[(past + j) * H];
  }
}

constexpr int RT_SMEM = 200 * 1024;

template <typename T, int N, bool WIDE>
static int launch_row_tiles(const RowTiles& a, dim3 grid, int threads, int smem, cudaStream_t s) {
  auto kern = row_tiles_kernel<T, N, WIDE>;
  if (smem > 48 * 1024) {
    static bool done = false;
    if (!done) { cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, RT_SMEM); done = true; }
  }
  spark_launch_pdl(kern, grid, dim3(threads), smem, s, dim3(1, 1, 1), a);
  return spark_launch_rc("spark_row_tiles");
}

}  // namespace spark

using namespace spark;

// nseg segments of at most max_rows rows (segs null: one of R rows); threads: at most so many per CTA.  -6: a row and its ring do not
// fit shared memory.
extern "C" int spark_row_tiles(const RowTiles* p, int nseg, int max_rows, int threads, int f32, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  const RowTiles& a = *p;
  const RowUpdate& u = a.u;
  const int H = u.H, past = a.taps > 1 ? a.taps - 1 : 0;
  if (H <= 0 || !u.res || u.post_w || u.norm < 0 || u.norm > 1 || (u.norm && !u.w) || a.groups < 1 || H % a.groups) return -5;
  if ((u.y && (u.slots <= 0 || !u.ids)) || (u.self_w && !u.self_x) || (a.stack && (!a.avg || a.k < 0))) return -5;
  if ((u.delta || u.y || a.stack) && (!a.res_out || a.res_out == u.res)) return -5;
  if (a.taps < 0 || (a.taps > 0 && (!a.conv_w || !a.segs)) || (past > 0 && !a.tail) || a.tile < 1 || a.tile < past || nseg > 65535) return -5;
  const uintptr_t al = reinterpret_cast<uintptr_t>(u.res) | reinterpret_cast<uintptr_t>(u.delta) | reinterpret_cast<uintptr_t>(u.y) |
                       reinterpret_cast<uintptr_t>(u.shared) | reinterpret_cast<uintptr_t>(u.self_x) | reinterpret_cast<uintptr_t>(u.scale) |
                       reinterpret_cast<uintptr_t>(u.w) | reinterpret_cast<uintptr_t>(u.out) | reinterpret_cast<uintptr_t>(u.out32) |
                       reinterpret_cast<uintptr_t>(a.res_out) | reinterpret_cast<uintptr_t>(a.stack) | reinterpret_cast<uintptr_t>(a.conv_w) |
                       reinterpret_cast<uintptr_t>(a.tail) | reinterpret_cast<uintptr_t>(a.rows);
  const int gs = H / a.groups, n = (al & 15) == 0 && (gs & 3) == 0 ? 4 : 1;
  const bool wide = n == 4 && (gs & 127) == 0;
  const int red = wide ? 3 * (H / 128) : H / n + a.groups;
  const size_t smem = (static_cast<size_t>(past + 1) * H + red) * 4;
  if (smem > RT_SMEM) return -6;
  const int want = (H / n + 31) / 32 * 32, most = threads < 32 ? 32 : (threads > 1024 ? 1024 : threads / 32 * 32);
  const int nt = want < most ? want : most;
  const dim3 grid((max_rows + a.tile - 1) / a.tile, nseg);
#define SPARK_TILES(T)                                                                   \
  return wide ? launch_row_tiles<T, 4, true>(a, grid, nt, static_cast<int>(smem), s)     \
       : n == 4 ? launch_row_tiles<T, 4, false>(a, grid, nt, static_cast<int>(smem), s)  \
                : launch_row_tiles<T, 1, false>(a, grid, nt, static_cast<int>(smem), s);
  if (f32) { SPARK_TILES(float) } else { SPARK_TILES(__nv_bfloat16) }
#undef SPARK_TILES
}

extern "C" int spark_tail_advance(float* tail, const float* rows, const int* segs, int nseg, const int* n_rows, int past, int H,
                                  cudaStream_t s) {
  if (nseg <= 0 || past <= 0) return 0;
  if (nseg > 65535) return -5;
  spark_launch_pdl(tail_advance_kernel, dim3((H + 255) / 256, nseg), dim3(256), 0, s, dim3(1, 1, 1), tail, rows, segs, n_rows, past, H);
  return spark_launch_rc(__func__);
}
