// Row kernels of designs that put a short causal convolution over time between a projection or a norm
// and what reads it.  Both walk tiles of kConvTile consecutive tokens of one batch entry: a thread owns
// VEC channels and keeps the last taps-1 inputs of each in registers, so an input is read once per tile.
// The inputs before a tile come from the batch (the entry's earlier rows), before the portion from the
// sequence's state row ([taps-1, channels] fp32, oldest first), before position 0 they are zero.  The
// CTA of a portion's FIRST tile is the only one that touches the state: it reads it before its walk and
// afterwards replaces it with the portion's last taps-1 inputs (read from the portion's end), so one
// launch needs no second pass and no CTA waits for another.
//
//   residual_norm_conv : y = x + a + b (fp32; terms optional), written to a second residual buffer;
//                        r = 1 / sqrt(mean(y^2) + eps);  h = y * r * w1;
//                        out1 = h + sum_j cw[j] * h_(t - taps + 1 + j)   (no taps: out1 = h)
//                        out2 = y * r * w2                                (optional second norm)
//                        = residual add, two pre-norms of the same residual and the mixer's input
//                        convolution of a parallel block in one launch.
//   conv_rot_write     : the projections [q | k | v] of a token, convolved; q and k then rotated (half
//                        pairing: coordinate i with i + rot/2 of every head map) by position x frequency;
//                        q out as fp32 and / or 16-bit rows, k and v into the token's pool row.
// Norms, convolutions, angles and rotation are fp32.
#include <type_traits>

#include "common.cuh"

namespace b200 {

constexpr int kConvTile = 16;        // tokens per CTA
constexpr int kConvThreads_ = 256;
constexpr int kMaxTaps = 16;

template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 lo = unpack2<T>(u.x), hi = unpack2<T>(u.y);
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
  } else if constexpr (VEC == 4) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = to_float<T>(p[e]);
  }
}

// A piece as it lies in memory, for loads that are requested rows ahead of their use
template <typename T, int VEC>
struct Piece {
  typename std::conditional<VEC == 4, typename std::conditional<sizeof(T) == 2, uint2, float4>::type, T>::type raw;
  __device__ __forceinline__ void load(const T* p) { raw = *reinterpret_cast<const decltype(raw)*>(p); }
  __device__ __forceinline__ void get(float (&v)[VEC]) const { load_vec<T, VEC>(reinterpret_cast<const T*>(&raw), v); }
};

template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 2) {
    alignas(8) T t[4] = {from_float<T>(v[0]), from_float<T>(v[1]), from_float<T>(v[2]), from_float<T>(v[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(t);
  } else if constexpr (VEC == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) p[e] = from_float<T>(v[e]);
  }
}

// the last MT - 1 inputs of a channel, newest at [MT - 2]; k tokens back is h[MT - 1 - k]
template <int MT, int VEC>
struct History {
  float h[MT - 1][VEC];
  __device__ __forceinline__ void clear() {
#pragma unroll
    for (int i = 0; i < MT - 1; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[i][e] = 0.f;
  }
  __device__ __forceinline__ void push(const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i + 1 < MT - 1; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[i][e] = h[i + 1][e];
#pragma unroll
    for (int e = 0; e < VEC; ++e) h[MT - 2][e] = v[e];
  }
  // state rows 0 .. taps-2 (oldest first) are the newest taps-1 entries
  __device__ __forceinline__ void from_state(const float* st, int64_t stride, int taps) {
#pragma unroll
    for (int i = 0; i < MT - 1; ++i) {
      const int s = i - (MT - taps);
      if (s >= 0) {
        float v[VEC];
        load_vec<float, VEC>(st + s * stride, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) h[i][e] = v[e];
      }
    }
  }
  __device__ __forceinline__ void to_state(float* st, int64_t stride, int taps) const {
#pragma unroll
    for (int i = 0; i < MT - 1; ++i) {
      const int s = i - (MT - taps);
      if (s >= 0) store_vec<float, VEC>(st + s * stride, h[i]);
    }
  }
};

// weight of the input k tokens back (cw [taps, C]: row j multiplies the input taps-1-j tokens back)
template <int MT, int VEC>
__device__ __forceinline__ void load_taps(const float* cw, int64_t C, int c, int taps, float (&wk)[MT][VEC]) {
#pragma unroll
  for (int k = 0; k < MT; ++k) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) wk[k][e] = 0.f;
    if (cw && k < taps) load_vec<float, VEC>(cw + (taps - 1 - k) * C + c, wk[k]);
  }
}

template <int MT, int VEC>
__device__ __forceinline__ void convolve(const float (&wk)[MT][VEC], const float (&v)[VEC],
                                         const History<MT, VEC>& hist, float (&y)[VEC]) {
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    float acc = wk[0][e] * v[e];
#pragma unroll
    for (int k = 1; k < MT; ++k) acc = fmaf(wk[k][e], hist.h[MT - 1 - k][e], acc);
    y[e] = acc;
  }
}

struct NormConvArgs {
  const float* x;
  int64_t ldx;
  const void *a, *b;
  int64_t lda, ldb;
  float* x_out;
  int64_t ldxo;
  const float *w1, *w2;
  float eps;
  const float* cw;
  int taps;
  float* state;
  int64_t ld_state;
  const int64_t* slot;
  const int *tok_pos, *ext_start, *ext_len;
  void *out1, *out2;
  int64_t ld1, ld2;
  int W;
};

template <typename T, int VEC, int MT>
__global__ void __launch_bounds__(kConvThreads_)
residual_norm_conv_kernel(const NormConvArgs p) {
  __shared__ float inv_s[kConvTile + 2 * (MT - 1)];
  __shared__ float red[kConvThreads_ / 32];
  const int bq = blockIdx.y, i0 = blockIdx.x * kConvTile, n = p.ext_len[bq];
  if (i0 >= n) return;
  const int r0 = p.ext_start[bq], m = min(kConvTile, n - i0), taps = p.taps, W = p.W;
  const bool first = i0 == 0;
  const int halo = first ? 0 : taps - 1;                    // i0 >= kConvTile >= taps - 1: all in the batch
  const int tail = first && n > kConvTile && p.state ? taps - 1 : 0;
  const int rows = halo + m + tail;
  // rows of the pass: the halo, the tile, then the portion's last rows (first tile of a longer portion)
  auto row_of = [&](int q) { return q < halo + m ? r0 + i0 - halo + q : r0 + n - tail + (q - halo - m); };
  const T* pa = static_cast<const T*>(p.a);
  const T* pb = static_cast<const T*>(p.b);
  auto load_row = [&](int64_t row, int c, float (&v)[VEC]) {
    load_vec<float, VEC>(p.x + row * p.ldx + c, v);
    if (pa) {
      float t[VEC];
      load_vec<T, VEC>(pa + row * p.lda + c, t);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] += t[e];
    }
    if (pb) {
      float t[VEC];
      load_vec<T, VEC>(pb + row * p.ldb + c, t);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] += t[e];
    }
  };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int NWARP = kConvThreads_ / 32;
  if (rows >= NWARP / 2) {                                  // a warp per row
    for (int q = warp; q < rows; q += NWARP) {
      const int64_t row = row_of(q);
      float s = 0.f;
#pragma unroll 4
      for (int c = lane * VEC; c < W; c += 32 * VEC) {
        float v[VEC];
        load_row(row, c, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s = fmaf(v[e], v[e], s);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (lane == 0) inv_s[q] = 1.0f / sqrtf(s / static_cast<float>(W) + p.eps);
    }
  } else {                                                  // a decoded token: the whole CTA per row
    for (int q = 0; q < rows; ++q) {
      const int64_t row = row_of(q);
      float s = 0.f;
      for (int c = threadIdx.x * VEC; c < W; c += kConvThreads_ * VEC) {
        float v[VEC];
        load_row(row, c, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s = fmaf(v[e], v[e], s);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      __syncthreads();
      if (lane == 0) red[warp] = s;
      __syncthreads();
      if (threadIdx.x == 0) {
        float t = 0.f;
        for (int w = 0; w < NWARP; ++w) t += red[w];
        inv_s[q] = 1.0f / sqrtf(t / static_cast<float>(W) + p.eps);
      }
    }
  }
  __syncthreads();
  float* st = p.state ? p.state + p.slot[bq] * p.ld_state : nullptr;
  const bool carried = first && st && p.tok_pos[r0] > 0;
  T* o1 = static_cast<T*>(p.out1);
  T* o2 = static_cast<T*>(p.out2);
  for (int c = threadIdx.x * VEC; c < W; c += kConvThreads_ * VEC) {
    float w1[VEC], w2[VEC], wk[MT][VEC];
    load_vec<float, VEC>(p.w1 + c, w1);
    if (o2) load_vec<float, VEC>(p.w2 + c, w2);
    load_taps<MT, VEC>(p.cw, W, c, taps, wk);
    History<MT, VEC> hist;
    hist.clear();
    if (carried) hist.from_state(st + c, W, taps);
    auto normed = [&](int q, float (&v)[VEC], float (&h)[VEC]) {
      load_row(row_of(q), c, v);
      const float r = inv_s[q];
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[e] = v[e] * r * w1[e];
    };
    for (int q = 0; q < halo; ++q) {
      float v[VEC], h[VEC];
      normed(q, v, h);
      hist.push(h);
    }
    // rows in batches: all loads of a batch are requested before its first row is used and stored
    constexpr int RB = MT <= 4 ? 4 : 1;
    for (int q0 = halo; q0 < halo + m; q0 += RB) {
      Piece<float, VEC> px[RB];
      Piece<T, VEC> ta[RB], tb[RB];
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const int64_t row = r0 + i0 + min(q0 + i - halo, m - 1);
        px[i].load(p.x + row * p.ldx + c);
        if (pa) ta[i].load(pa + row * p.lda + c);
        if (pb) tb[i].load(pb + row * p.ldb + c);
      }
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const int q = q0 + i;
        if (q >= halo + m) break;
        const int64_t row = r0 + i0 + (q - halo);
        const float r = inv_s[q];
        float v[VEC], h[VEC], y[VEC];
        px[i].get(v);
        if (pa) {
          ta[i].get(h);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[e] += h[e];
        }
        if (pb) {
          tb[i].get(h);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[e] += h[e];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) h[e] = v[e] * r * w1[e];
        convolve<MT, VEC>(wk, h, hist, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] += h[e];
        hist.push(h);
        store_vec<float, VEC>(p.x_out + row * p.ldxo + c, v);
        store_vec<T, VEC>(o1 + row * p.ld1 + c, y);
        if (o2) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[e] = v[e] * r * w2[e];
          store_vec<T, VEC>(o2 + row * p.ld2 + c, y);
        }
      }
    }
    if (first && st) {
      for (int q = halo + m; q < rows; ++q) {
        float v[VEC], h[VEC];
        normed(q, v, h);
        hist.push(h);
      }
      hist.to_state(st + c, W, taps);
    }
  }
}

struct ConvRotArgs {
  const void* y;
  int64_t ldy;
  const float* cw;
  int taps;
  float* state;
  int64_t ld_state;
  const int64_t* slot;
  const int *tok_pos, *ext_start, *ext_len;
  const float *freq_hi, *freq_lo;
  int rot;
  const int64_t* loc;
  void* pool;
  int64_t ld_pool;
  int k_off, v_off;
  float* q32;
  int64_t ldq32;
  void* q16;
  int64_t ldq16;
  int NQ, NK, D, NV;          // query maps, key maps, map size, value channels
};

template <typename T, int VEC, int MT>
__global__ void __launch_bounds__(kConvThreads_)
conv_rot_write_kernel(const ConvRotArgs p) {
  extern __shared__ float cr_smem[];                        // [kConvTile][half] cos, then sin
  const int bq = blockIdx.y, i0 = blockIdx.x * kConvTile, n = p.ext_len[bq];
  if (i0 >= n) return;
  const int r0 = p.ext_start[bq], m = min(kConvTile, n - i0), taps = p.taps;
  const int D = p.D, half = p.rot / 2;
  float* cs = cr_smem;
  float* sn = cr_smem + kConvTile * half;
  const int pos0 = p.tok_pos[r0];
  for (int i = threadIdx.x; i < m * half; i += blockDim.x) {
    const int q = i / half, f = i - q * half;
    const float pos = static_cast<float>(pos0 + i0 + q);
    const float hi = p.freq_hi[f], lo = p.freq_lo[f];
    const float ang = pos * hi;
    const float err = fmaf(pos, hi, -ang) + pos * lo;       // what the rounded product dropped
    float s, c;
    sincosf(ang, &s, &c);
    cs[i] = c - err * s;
    sn[i] = s + err * c;
  }
  __syncthreads();
  const int NM = p.NQ + p.NK, C = NM * D + p.NV;
  const int rot_units = half / VEC, upm = rot_units + (D - p.rot + 2 * VEC - 1) / (2 * VEC);
  const int v_units = (p.NV + 2 * VEC - 1) / (2 * VEC);
  const int unit = blockIdx.z * blockDim.x + threadIdx.x;
  if (unit >= NM * upm + v_units) return;
  // a unit is two pieces of VEC channels: the two halves of rotated pairs, or neighbours
  int ca, cb, f0 = 0;
  bool rotated = false, live_b;
  if (unit < NM * upm) {
    const int map = unit / upm, u = unit - map * upm;
    if (u < rot_units) {
      rotated = true;
      f0 = u * VEC;
      ca = map * D + f0;
      cb = ca + half;
      live_b = true;
    } else {
      ca = map * D + p.rot + (u - rot_units) * 2 * VEC;
      cb = ca + VEC;
      live_b = cb < (map + 1) * D;
    }
  } else {
    ca = NM * D + (unit - NM * upm) * 2 * VEC;
    cb = ca + VEC;
    live_b = cb < C;
  }
  if (!live_b) cb = ca;                                     // a valid address; the result is not stored
  const T* yin = static_cast<const T*>(p.y);
  float wa[MT][VEC], wb[MT][VEC];
  load_taps<MT, VEC>(p.cw, C, ca, taps, wa);
  load_taps<MT, VEC>(p.cw, C, cb, taps, wb);
  History<MT, VEC> ha, hb;
  ha.clear();
  hb.clear();
  float* st = p.state ? p.state + p.slot[bq] * p.ld_state : nullptr;
  const bool first = i0 == 0;
  if (first) {
    if (st && pos0 > 0) {
      ha.from_state(st + ca, C, taps);
      hb.from_state(st + cb, C, taps);
    }
  } else {
    for (int q = -(taps - 1); q < 0; ++q) {
      float va[VEC], vb[VEC];
      const int64_t row = r0 + i0 + q;
      load_vec<T, VEC>(yin + row * p.ldy + ca, va);
      load_vec<T, VEC>(yin + row * p.ldy + cb, vb);
      ha.push(va);
      hb.push(vb);
    }
  }
  const int cq = p.NQ * D, ck = NM * D;
  T* pool = static_cast<T*>(p.pool);
  T* q16 = static_cast<T*>(p.q16);
  auto put = [&](int64_t row, int64_t prow, int c, const float (&v)[VEC]) {
    if (c < cq) {
      if (p.q32) store_vec<float, VEC>(p.q32 + row * p.ldq32 + c, v);
      if (q16) store_vec<T, VEC>(q16 + row * p.ldq16 + c, v);
    } else {
      store_vec<T, VEC>(pool + prow * p.ld_pool + (c < ck ? p.k_off + c - cq : p.v_off + c - ck), v);
    }
  };
  constexpr int RB = MT <= 4 ? 4 : 1;                       // rows requested together
  for (int q0 = 0; q0 < m; q0 += RB) {
    Piece<T, VEC> pa[RB], pb[RB];
    int64_t prow[RB];
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int64_t row = r0 + i0 + min(q0 + i, m - 1);
      pa[i].load(yin + row * p.ldy + ca);
      pb[i].load(yin + row * p.ldy + cb);
      prow[i] = ca >= cq ? p.loc[row] : 0;
    }
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int q = q0 + i;
      if (q >= m) break;
      const int64_t row = r0 + i0 + q;
      float va[VEC], vb[VEC], ya[VEC], yb[VEC];
      pa[i].get(va);
      pb[i].get(vb);
      if (p.cw) {
        convolve<MT, VEC>(wa, va, ha, ya);
        convolve<MT, VEC>(wb, vb, hb, yb);
        ha.push(va);
        hb.push(vb);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          ya[e] = va[e];
          yb[e] = vb[e];
        }
      }
      if (rotated) {
        float c[VEC], s[VEC];
        load_vec<float, VEC>(cs + q * half + f0, c);
        load_vec<float, VEC>(sn + q * half + f0, s);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const float u = ya[e], v = yb[e];
          ya[e] = fmaf(u, c[e], -v * s[e]);
          yb[e] = fmaf(v, c[e], u * s[e]);
        }
      }
      put(row, prow[i], ca, ya);
      if (live_b) put(row, prow[i], cb, yb);
    }
  }
  if (first && st) {
    if (n > kConvTile) {                                    // the portion goes on past this tile
      for (int q = n - (taps - 1); q < n; ++q) {
        float va[VEC], vb[VEC];
        const int64_t row = r0 + q;
        load_vec<T, VEC>(yin + row * p.ldy + ca, va);
        load_vec<T, VEC>(yin + row * p.ldy + cb, vb);
        ha.push(va);
        hb.push(vb);
      }
    }
    ha.to_state(st + ca, C, taps);
    if (live_b) hb.to_state(st + cb, C, taps);
  }
}

template <typename T>
static bool vec_ok(const void* p, int64_t ld) {
  return !p || (reinterpret_cast<uintptr_t>(p) % (4 * sizeof(T)) == 0 && ld % 4 == 0);
}

template <typename T>
static int launch_norm_conv(const NormConvArgs& p, int bs, int max_ext, cudaStream_t st) {
  const dim3 grid(ceil_div(max_ext, kConvTile), bs);
  const bool vec = p.W % 4 == 0 && vec_ok<float>(p.x, p.ldx) && vec_ok<T>(p.a, p.lda) && vec_ok<T>(p.b, p.ldb) &&
                   vec_ok<float>(p.x_out, p.ldxo) && vec_ok<float>(p.w1, 4) && vec_ok<float>(p.w2, 4) &&
                   vec_ok<float>(p.cw, 4) && vec_ok<float>(p.state, p.ld_state) && vec_ok<T>(p.out1, p.ld1) &&
                   vec_ok<T>(p.out2, p.ld2);
  ScopedKernelTimer timer("residual_norm_conv", st);
#define LAUNCH(V, M) \
  launch_kernel(residual_norm_conv_kernel<T, V, M>, grid, dim3(kConvThreads_), 0, st, 1, 0, p)
  if (p.taps > 4) LAUNCH(1, kMaxTaps);
  else if (vec) LAUNCH(4, 4);
  else LAUNCH(1, 4);
#undef LAUNCH
  B200_CHECK_LAUNCH("residual_norm_conv_kernel");
  return 0;
}

template <typename T>
static int launch_conv_rot(const ConvRotArgs& p, int bs, int max_ext, cudaStream_t st) {
  const bool vec = p.taps <= 4 && p.D % 4 == 0 && p.rot % 8 == 0 && p.NV % 4 == 0 && vec_ok<T>(p.y, p.ldy) &&
                   vec_ok<float>(p.cw, 4) && vec_ok<float>(p.state, p.ld_state) && vec_ok<T>(p.pool, p.ld_pool) &&
                   p.k_off % 4 == 0 && p.v_off % 4 == 0 && vec_ok<float>(p.q32, p.ldq32) && vec_ok<T>(p.q16, p.ldq16);
  const int V = vec ? 4 : 1;
  const int units = (p.NQ + p.NK) * (p.rot / 2 / V + ceil_div(p.D - p.rot, 2 * V)) + ceil_div(p.NV, 2 * V);
  int threads = ceil_div(units, 32) * 32;
  // enough CTAs for a few decoded tokens to spread over the machine
  const int cap = max_ext == 1 ? 64 : kConvThreads_;
  threads = threads < cap ? threads : cap;
  const dim3 grid(ceil_div(max_ext, kConvTile), bs, ceil_div(units, threads));
  const size_t smem = sizeof(float) * kConvTile * p.rot;
  ScopedKernelTimer timer("conv_rot_write", st);
#define LAUNCH(V_, M) launch_kernel(conv_rot_write_kernel<T, V_, M>, grid, dim3(threads), smem, st, 1, 0, p)
  if (p.taps > 4) LAUNCH(1, kMaxTaps);
  else if (vec) LAUNCH(4, 4);
  else LAUNCH(1, 4);
#undef LAUNCH
  B200_CHECK_LAUNCH("conv_rot_write_kernel");
  return 0;
}

}  // namespace b200

extern "C" int b200_residual_norm_conv(const float* x, int64_t ldx, const void* a, int64_t lda,
                                       const void* b, int64_t ldb, float* x_out, int64_t ldxo,
                                       const float* w1, const float* w2, float eps, const float* cw,
                                       int taps, float* state, int64_t ld_state, const int64_t* slot,
                                       const int* tok_pos, const int* ext_start, const int* ext_len,
                                       void* out1, int64_t ld1, void* out2, int64_t ld2, int bs,
                                       int max_ext, int W, int dtype, void* stream) {
  using namespace b200;
  if (bs == 0 || max_ext == 0) return 0;
  B200_REQUIRE(x && x_out && x != x_out && w1 && out1 && slot && tok_pos && ext_start && ext_len && (!out2 || w2),
               "b200_residual_norm_conv: null pointer, or the residual written in place");
  B200_REQUIRE(bs > 0 && bs <= 65535 && max_ext > 0 && W > 0 && taps >= 1 && taps <= kMaxTaps,
               "b200_residual_norm_conv: %d entries, %d taps (1 to %d)", bs, taps, kMaxTaps);
  B200_REQUIRE(taps == 1 || (cw && state), "b200_residual_norm_conv: a convolution needs weights and state rows");
  NormConvArgs p{x, ldx, a, b, lda, ldb, x_out, ldxo, w1, w2, eps, cw, taps, taps > 1 ? state : nullptr, ld_state,
                 slot, tok_pos, ext_start, ext_len, out1, out2, ld1, ld2, W};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B200_BF16) return launch_norm_conv<__nv_bfloat16>(p, bs, max_ext, st);
  if (dtype == B200_F16) return launch_norm_conv<__half>(p, bs, max_ext, st);
  if (dtype == B200_F32) return launch_norm_conv<float>(p, bs, max_ext, st);
  B200_REQUIRE(false, "b200_residual_norm_conv: dtype %d", dtype);
}

extern "C" int b200_conv_rot_write(const void* y, int64_t ldy, const float* cw, int taps, float* state,
                                   int64_t ld_state, const int64_t* slot, const int* tok_pos,
                                   const int* ext_start, const int* ext_len, const float* freq_hi,
                                   const float* freq_lo, int rot_dims, const int64_t* loc, void* pool,
                                   int64_t ld_pool, int k_off, int v_off, float* q32, int64_t ldq32,
                                   void* q16, int64_t ldq16, int q_maps, int k_maps, int D,
                                   int v_channels, int bs, int max_ext, int dtype, void* stream) {
  using namespace b200;
  if (bs == 0 || max_ext == 0) return 0;
  B200_REQUIRE(y && slot && tok_pos && ext_start && ext_len && (q32 || q16 || q_maps == 0) &&
                   ((k_maps == 0 && v_channels == 0) || (pool && loc)),
               "b200_conv_rot_write: null pointer");
  B200_REQUIRE(bs > 0 && bs <= 65535 && max_ext > 0 && taps >= 1 && taps <= kMaxTaps && q_maps >= 0 && k_maps >= 0 &&
                   v_channels >= 0 && D > 0 && q_maps + k_maps + v_channels > 0,
               "b200_conv_rot_write: %d entries, %d taps (1 to %d), maps %d / %d of %d", bs, taps, kMaxTaps, q_maps,
               k_maps, D);
  B200_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= D && rot_dims <= 512 &&
                   (rot_dims == 0 || (freq_hi && freq_lo)),
               "b200_conv_rot_write: %d of %d coordinates rotated", rot_dims, D);
  B200_REQUIRE(taps == 1 || (cw && state), "b200_conv_rot_write: a convolution needs weights and state rows");
  ConvRotArgs p{y, ldy, cw, taps, taps > 1 ? state : nullptr, ld_state, slot, tok_pos, ext_start, ext_len, freq_hi,
                freq_lo, rot_dims, loc, pool, ld_pool, k_off, v_off, q32, ldq32, q16, ldq16, q_maps, k_maps, D,
                v_channels};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B200_BF16) return launch_conv_rot<__nv_bfloat16>(p, bs, max_ext, st);
  if (dtype == B200_F16) return launch_conv_rot<__half>(p, bs, max_ext, st);
  if (dtype == B200_F32) return launch_conv_rot<float>(p, bs, max_ext, st);
  B200_REQUIRE(false, "b200_conv_rot_write: dtype %d", dtype);
}
