// The channel-gated memory of linear_recurrence.cu (S_t = diag(f_t) S_(t-1) + w_t v_t^T, w = 1 - f,
// o_t = S_t^T q_t) for long prompt portions, 16 tokens at a time.  Within a chunk that starts from S_0, with
// f_(a,b] = prod_{a < s <= b} f_s per channel:
//
//   o_i  = (q_i f_(0,i])^T S_0 + sum_{j <= i} A_ij v_j,      A_ij = sum_d q_i[d] w_j[d] f_(j,i][d]
//   S_16 = diag(f_(0,16]) S_0 + sum_j (w_j f_(j,16]) v_j^T
//
// Every factor is a product of gates between 0 and 1 that is formed as a product (never as a quotient of
// running products), so nothing overflows however little a gate keeps, and everything is fp32.
//
//   channel_prepare : one CTA per (chunk, head), all chunks in parallel: the gates and activations, the rows
//                     q f_(0,i] and w f_(j,16], the chunk's decay, and A.  A lane owns D / 32 channels of all 16
//                     tokens in registers; a warp takes every fourth j, and the 16 sums of one j are reduced
//                     over the lanes together (each step halves the values a lane still carries).
//   channel_scan    : one warp owns 4 * 32 / (D / 8) value columns of a head for the whole portion; a lane holds
//                     8 channels x 4 columns of S in registers, channel pairs packed.  Per chunk: the 16 x 4
//                     partial outputs of its channels (the rows it needs come out of shared memory as pairs),
//                     reduced over the lanes of a column in the same halving way, so each lane ends with the
//                     row(s) it stores; then 16 rank-one updates.  No step of a chunk depends on another token's,
//                     so the work is multiply-adds from registers instead of a chain through the tokens.  The next
//                     chunk's rows stream in (cp.async) meanwhile.
//
// The state row is read and written in linear_recurrence.cu's layout: portions and single tokens alternate freely.
#include "f32x2.cuh"

namespace b200 {

constexpr int kChunk = 16;

struct ChunkArgs {
  const void *q, *zf, *v;
  int64_t ldq, ldf, ldv;
  const float *f_bias, *f_lower;
  float q_scale;
  int act, min_len;
  float* state;
  int64_t ld_state;
  const int64_t* slot;
  const int *tok_pos, *ext_start, *ext_len;
  float *wq, *wk, *wa, *wp;    // [T][H][Dp], [T][H][Dp], [chunk][H][16 j][16 i], [chunk][H][Dp]
  float* out;
  int64_t ldo;
  int H, D, E;
};

// chunk number c of batch entry b: ids of different entries do not meet, and stay below T / 16 + batch + 1
__device__ __forceinline__ int64_t chunk_id(int start, int b, int c) { return start / kChunk + b + c; }

// acc[x] of lanes that differ in bit `m` of the lane are added; the lane keeps the half its bit names
template <int HALF>
__device__ __forceinline__ void halve(float* acc, int m, bool upper) {
#pragma unroll
  for (int x = 0; x < HALF; ++x) {
    const float send = upper ? acc[x] : acc[x + HALF];
    const float keep = upper ? acc[x + HALF] : acc[x];
    acc[x] = keep + __shfl_xor_sync(0xffffffffu, send, m);
  }
}

template <typename T, int CPL>
__global__ void __launch_bounds__(128)
channel_prepare_kernel(const ChunkArgs a) {
  constexpr int Dp = 32 * CPL;
  __shared__ __align__(16) float qs[kChunk][Dp], ws[kChunk][Dp];
  const int b = blockIdx.z, h = blockIdx.y, len = a.ext_len[b];
  const int c0 = blockIdx.x * kChunk;
  if (len < a.min_len || c0 >= len) return;
  const int n = min(kChunk, len - c0);
  const int start = a.ext_start[b];
  const int64_t row0 = start + c0, cid = chunk_id(start, b, blockIdx.x);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, d0 = lane * CPL;
  float lo[CPL], bi[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const bool in = d0 + c < a.D;
    lo[c] = in && a.f_lower ? a.f_lower[h * a.D + d0 + c] : 0.f;
    bi[c] = in && a.f_bias ? a.f_bias[h * a.D + d0 + c] : 0.f;
  }
  const T* qg = static_cast<const T*>(a.q) + h * a.D + d0;
  const T* zg = static_cast<const T*>(a.zf) + h * a.D + d0;
  float qr[kChunk / 4][CPL], zr[kChunk / 4][CPL];
#pragma unroll
  for (int k = 0; k < kChunk / 4; ++k) {       // the warp's tokens: all loads requested before the first use
    const int i = warp + 4 * k;
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const bool in = i < n && d0 + c < a.D;
      qr[k][c] = in ? to_float<T>(qg[(row0 + i) * a.ldq + c]) : 0.f;
      zr[k][c] = in ? to_float<T>(zg[(row0 + i) * a.ldf + c]) : 0.f;
    }
  }
#pragma unroll
  for (int k = 0; k < kChunk / 4; ++k) {
    const int i = warp + 4 * k;
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const bool in = i < n && d0 + c < a.D;
      const float q = qr[k][c];
      qs[i][d0 + c] = (a.act == 1 ? q / (1.0f + expf(-q)) : q) * a.q_scale;
      ws[i][d0 + c] = in ? (1.0f - lo[c]) / (1.0f + expf(zr[k][c] + bi[c])) : 0.f;   // the written share
    }
  }
  __syncthreads();
  float q[kChunk][CPL], f[kChunk][CPL];
#pragma unroll
  for (int i = 0; i < kChunk; ++i)
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      q[i][c] = qs[i][d0 + c];
      f[i][c] = 1.0f - ws[i][d0 + c];
    }
  auto put = [&](float* dst, const float (&x)[CPL]) {
    if constexpr (CPL == 4) *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
    else if constexpr (CPL == 2) *reinterpret_cast<float2*>(dst) = make_float2(x[0], x[1]);
    else dst[0] = x[0];
  };
  float p[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) p[c] = 1.f;
#pragma unroll
  for (int i = 0; i < kChunk; ++i) {
    float y[CPL];
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      p[c] *= f[i][c];
      y[c] = q[i][c] * p[c];
    }
    if ((i & 3) == warp && i < n) put(a.wq + ((row0 + i) * a.H + h) * Dp + d0, y);
  }
  if (warp == 0) put(a.wp + (cid * a.H + h) * Dp + d0, p);
#pragma unroll
  for (int c = 0; c < CPL; ++c) p[c] = 1.f;
#pragma unroll
  for (int j = kChunk - 1; j >= 0; --j) {
    if ((j & 3) == warp && j < n) {
      float y[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) y[c] = ws[j][d0 + c] * p[c];
      put(a.wk + ((row0 + j) * a.H + h) * Dp + d0, y);
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c) p[c] *= f[j][c];
  }
  float* A = a.wa + (cid * a.H + h) * (kChunk * kChunk);
#pragma unroll 1
  for (int j = warp; j < kChunk; j += 4) {
    float part[kChunk];
#pragma unroll
    for (int c = 0; c < CPL; ++c) p[c] = ws[j][d0 + c];
#pragma unroll
    for (int i = 0; i < kChunk; ++i) {
      part[i] = 0.f;
      if (i >= j) {
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          if (i > j) p[c] *= f[i][c];
          part[i] = fmaf(q[i][c], p[c], part[i]);
        }
      }
    }
    halve<8>(part, 16, lane & 16);
    halve<4>(part, 8, lane & 8);
    halve<2>(part, 4, lane & 4);
    halve<1>(part, 2, lane & 2);
    part[0] += __shfl_xor_sync(0xffffffffu, part[0], 1);
    if (!(lane & 1)) A[j * kChunk + (lane >> 1)] = part[0];
  }
}

// LPD lanes share a column group: Dp = 8 * LPD channels
template <typename T, int LPD>
__global__ void __launch_bounds__(128)
channel_scan_kernel(const ChunkArgs a) {
  constexpr int Dp = 8 * LPD, CW = 4 * (32 / LPD), JL = kChunk / LPD;   // columns per warp; rows i, j per lane
  extern __shared__ __align__(16) float cs_smem[];
  const int b = blockIdx.z, h = blockIdx.y, len = a.ext_len[b];
  if (len < a.min_len) return;
  const int NT = blockDim.x, ES = (NT >> 5) * CW, e0 = blockIdx.x * ES;
  const int start = a.ext_start[b], E = a.E, H = a.H;
  const bool fresh = a.tok_pos[start] == 0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane % LPD, cl = warp * CW + (lane / LPD) * 4, e = e0 + cl;
  // one stage: q [16][Dp], k [16][Dp], A [16 j][16 i], decay [Dp], v [16][ES] (in T, padded to 16 bytes)
  const int v_at = 2 * kChunk * Dp + kChunk * kChunk + Dp;
  const int stage_floats = v_at + (kChunk * ES * static_cast<int>(sizeof(T)) + 15) / 16 * 4;
  for (int i = tid; i < 2 * stage_floats; i += NT) cs_smem[i] = 0.f;     // columns past E stay zero
  __syncthreads();
  const T* vg = static_cast<const T*>(a.v) + h * E + e0;
  const int nc = min(ES, E - e0);              // columns of this slice that exist
  constexpr int PV = 8 / sizeof(T);
  const bool v_async = (reinterpret_cast<uintptr_t>(vg) & 7) == 0 && a.ldv % PV == 0 && nc % PV == 0;
  auto stage = [&](int c, float* buf) {
    const int c0 = c * kChunk, n = min(kChunk, len - c0);
    const int64_t row0 = start + c0, cid = chunk_id(start, b, c);
    for (int x = tid; x < 2 * kChunk * (Dp / 4); x += NT) {
      const int kind = x / (kChunk * (Dp / 4)), y = x - kind * (kChunk * (Dp / 4));
      const int i = y / (Dp / 4), d = (y - i * (Dp / 4)) * 4;
      float* dst = buf + kind * kChunk * Dp + i * Dp + d;
      if (i < n) cp_async16(smem_u32(dst), (kind ? a.wk : a.wq) + ((row0 + i) * H + h) * Dp + d);
      else *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int x = tid; x < kChunk * kChunk / 4 + Dp / 4; x += NT) {
      const int y = x - kChunk * kChunk / 4;
      if (y < 0) cp_async16(smem_u32(buf + 2 * kChunk * Dp + x * 4), a.wa + (cid * H + h) * (kChunk * kChunk) + x * 4);
      else cp_async16(smem_u32(buf + 2 * kChunk * Dp + kChunk * kChunk + y * 4), a.wp + (cid * H + h) * Dp + y * 4);
    }
    T* vs = reinterpret_cast<T*>(buf + v_at);
    if (v_async) {
      const int per = nc / PV;
      for (int x = tid; x < kChunk * per; x += NT) {
        const int i = x / per, col = (x - i * per) * PV;
        if (i < n)
          asm volatile("cp.async.ca.shared.global [%0], [%1], 8;\n" ::"r"(smem_u32(vs + i * ES + col)),
                       "l"(vg + (row0 + i) * a.ldv + col));
        else
          *reinterpret_cast<uint2*>(vs + i * ES + col) = make_uint2(0u, 0u);
      }
    } else {
      for (int x = tid; x < kChunk * nc; x += NT) {
        const int i = x / nc, col = x - i * nc;
        vs[i * ES + col] = i < n ? vg[(row0 + i) * a.ldv + col] : from_float<T>(0.f);
      }
    }
    cp_async_commit();
  };
  // state: atoms of 4 rows x 2 columns, [column pair][row / 4]
  const int NCP = (E + 1) / 2, D4 = (a.D + 3) / 4;
  float* st = a.state + a.slot[b] * a.ld_state + static_cast<int64_t>(h) * D4 * NCP * 8;
  f32x2 s[2][2][4];                            // [atom][row pair][column]
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int c2 = 0; c2 < 2; ++c2) {
      const int d4 = t * LPD + g, cp = e / 2 + c2;
      float4 v0 = make_float4(0.f, 0.f, 0.f, 0.f), v1 = v0;
      if (!fresh && d4 < D4 && cp < NCP) {
        const float4* at = reinterpret_cast<const float4*>(st + (static_cast<int64_t>(cp) * D4 + d4) * 8);
        v0 = at[0];
        v1 = at[1];
      }
      s[t][0][2 * c2] = pack2(v0.x, v0.z);
      s[t][0][2 * c2 + 1] = pack2(v0.y, v0.w);
      s[t][1][2 * c2] = pack2(v1.x, v1.z);
      s[t][1][2 * c2 + 1] = pack2(v1.y, v1.w);
    }
  const bool out_vec = E % 4 == 0 && a.ldo % 4 == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
  const int chunks = (len + kChunk - 1) / kChunk;
  auto values = [&](const T* vs, int j, float (&x)[4]) {      // this lane's 4 columns of row j
    const T* p = vs + j * ES + cl;
    if constexpr (sizeof(T) == 2) {
      const uint2 u = *reinterpret_cast<const uint2*>(p);
      const float2 lo = b200::unpack2<T>(u.x), hi = b200::unpack2<T>(u.y);
      x[0] = lo.x, x[1] = lo.y, x[2] = hi.x, x[3] = hi.y;
    } else {
      const float4 u = *reinterpret_cast<const float4*>(p);
      x[0] = u.x, x[1] = u.y, x[2] = u.z, x[3] = u.w;
    }
  };
  stage(0, cs_smem);
  for (int c = 0; c < chunks; ++c) {
    cp_async_wait<0>();
    __syncthreads();                           // chunk c is in; every warp has left chunk c - 1
    if (c + 1 < chunks) stage(c + 1, cs_smem + ((c + 1) & 1) * stage_floats);
    const float* buf = cs_smem + (c & 1) * stage_floats;
    const float *qs = buf, *ks = buf + kChunk * Dp, *As = ks + kChunk * Dp, *ps = As + kChunk * kChunk;
    const T* vs = reinterpret_cast<const T*>(buf + v_at);
    float vl[JL][4];                           // the rows j this lane contributes to the inner sums
#pragma unroll
    for (int k = 0; k < JL; ++k) values(vs, g + k * LPD, vl[k]);
    float part[kChunk * 4];
#pragma unroll
    for (int ig = 0; ig < kChunk / 4; ++ig) {
      f32x2 acc[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const ulonglong2 q0 = *reinterpret_cast<const ulonglong2*>(qs + (4 * ig + i) * Dp + 4 * g);
        const ulonglong2 q1 = *reinterpret_cast<const ulonglong2*>(qs + (4 * ig + i) * Dp + 4 * (LPD + g));
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          acc[i][x] = mul2(s[0][0][x], q0.x);
          acc[i][x] = fma2(s[0][1][x], q0.y, acc[i][x]);
          acc[i][x] = fma2(s[1][0][x], q1.x, acc[i][x]);
          acc[i][x] = fma2(s[1][1][x], q1.y, acc[i][x]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          float lo, hi;
          unpack2(acc[i][x], lo, hi);
          part[(4 * ig + i) * 4 + x] = lo + hi;
        }
#pragma unroll
      for (int k = 0; k < JL; ++k) {
        const float4 A4 = *reinterpret_cast<const float4*>(As + (g + k * LPD) * kChunk + 4 * ig);
        const float Ai[4] = {A4.x, A4.y, A4.z, A4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int x = 0; x < 4; ++x) part[(4 * ig + i) * 4 + x] = fmaf(Ai[i], vl[k][x], part[(4 * ig + i) * 4 + x]);
      }
    }
    // sum over the LPD lanes of a column group; the lane keeps rows g * JL ... g * JL + JL - 1
    if constexpr (LPD == 16) {
      halve<32>(part, 8, g & 8);
      halve<16>(part, 4, g & 4);
      halve<8>(part, 2, g & 2);
      halve<4>(part, 1, g & 1);
    } else if constexpr (LPD == 8) {
      halve<32>(part, 4, g & 4);
      halve<16>(part, 2, g & 2);
      halve<8>(part, 1, g & 1);
    } else {
      halve<32>(part, 2, g & 2);
      halve<16>(part, 1, g & 1);
    }
    const int n = min(kChunk, len - c * kChunk);
#pragma unroll
    for (int r = 0; r < JL; ++r) {
      const int i = g * JL + r;
      if (i < n && e < E) {
        float* dst = a.out + (start + c * kChunk + i) * a.ldo + h * E + e;
        if (out_vec) {
          *reinterpret_cast<float4*>(dst) = make_float4(part[r * 4], part[r * 4 + 1], part[r * 4 + 2], part[r * 4 + 3]);
        } else {
#pragma unroll
          for (int x = 0; x < 4; ++x)
            if (e + x < E) dst[x] = part[r * 4 + x];
        }
      }
    }
    // S <- diag(decay) S + sum_j k_j v_j^T
    {
      const ulonglong2 p0 = *reinterpret_cast<const ulonglong2*>(ps + 4 * g);
      const ulonglong2 p1 = *reinterpret_cast<const ulonglong2*>(ps + 4 * (LPD + g));
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        s[0][0][x] = mul2(s[0][0][x], p0.x);
        s[0][1][x] = mul2(s[0][1][x], p0.y);
        s[1][0][x] = mul2(s[1][0][x], p1.x);
        s[1][1][x] = mul2(s[1][1][x], p1.y);
      }
    }
#pragma unroll 4
    for (int j = 0; j < kChunk; ++j) {
      const ulonglong2 k0 = *reinterpret_cast<const ulonglong2*>(ks + j * Dp + 4 * g);
      const ulonglong2 k1 = *reinterpret_cast<const ulonglong2*>(ks + j * Dp + 4 * (LPD + g));
      float x4[4];
      values(vs, j, x4);
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const f32x2 vv = pack2(x4[x], x4[x]);
        s[0][0][x] = fma2(k0.x, vv, s[0][0][x]);
        s[0][1][x] = fma2(k0.y, vv, s[0][1][x]);
        s[1][0][x] = fma2(k1.x, vv, s[1][0][x]);
        s[1][1][x] = fma2(k1.y, vv, s[1][1][x]);
      }
    }
  }
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int c2 = 0; c2 < 2; ++c2) {
      const int d4 = t * LPD + g, cp = e / 2 + c2;
      if (d4 < D4 && cp < NCP) {
        float4* at = reinterpret_cast<float4*>(st + (static_cast<int64_t>(cp) * D4 + d4) * 8);
        float4 v0, v1;
        unpack2(s[t][0][2 * c2], v0.x, v0.z);
        unpack2(s[t][0][2 * c2 + 1], v0.y, v0.w);
        unpack2(s[t][1][2 * c2], v1.x, v1.z);
        unpack2(s[t][1][2 * c2 + 1], v1.y, v1.w);
        at[0] = v0;
        at[1] = v1;
      }
    }
}

static int chunk_lanes(int D) { return D <= 32 ? 4 : (D <= 64 ? 8 : 16); }

}  // namespace b200

// floats of workspace b200_channel_chunks needs (-1: key size not served)
extern "C" int64_t b200_channel_chunks_work(int T, int batch, int H, int D) {
  using namespace b200;
  if (T < 0 || batch < 0 || H <= 0 || D <= 0 || D > 128) return -1;
  const int64_t Dp = 8 * chunk_lanes(D), nchunks = T / kChunk + batch + 1;
  return 2 * static_cast<int64_t>(T) * H * Dp + nchunks * H * (kChunk * kChunk + Dp);
}

// The entries of at least min_len new tokens of the step, longest max_len; arguments as b200_channel_recurrence.
extern "C" int b200_channel_chunks(const void* q, int64_t ldq, const void* zf, int64_t ldf, const void* v,
                                   int64_t ldv, const float* f_bias, const float* f_lower, float q_scale, int act,
                                   float* state, int64_t ld_state, const int64_t* slot, const int* tok_pos,
                                   const int* ext_start, const int* ext_len, float* out, int64_t ldo, float* work,
                                   int T, int batch, int min_len, int max_len, int H, int D, int E, int dtype,
                                   void* stream) {
  using namespace b200;
  if (batch == 0 || T == 0 || max_len < min_len) return 0;
  B200_REQUIRE(q && zf && v && state && slot && tok_pos && ext_start && ext_len && out && work,
               "b200_channel_chunks: null pointer");
  B200_REQUIRE(T > 0 && batch > 0 && min_len > 0 && H > 0 && D > 0 && D <= 128 && E > 0 && (act == 0 || act == 1),
               "b200_channel_chunks: heads %d, key size %d (max 128), value size %d", H, D, E);
  B200_REQUIRE(ld_state % 4 == 0 && aligned16(state) && aligned16(work),
               "b200_channel_chunks: state rows and workspace must be 16-byte aligned");
  B200_REQUIRE(H <= 65535 && batch <= 65535, "b200_channel_chunks: grid too large");
  const int lpd = chunk_lanes(D), Dp = 8 * lpd, cw = 4 * (32 / lpd);
  const int64_t nchunks = T / kChunk + batch + 1;
  ChunkArgs a{q, zf, v, ldq, ldf, ldv, f_bias, f_lower, q_scale, act, min_len, state, ld_state, slot, tok_pos, ext_start,
              ext_len, work, nullptr, nullptr, nullptr, out, ldo, H, D, E};
  a.wk = a.wq + static_cast<int64_t>(T) * H * Dp;
  a.wa = a.wk + static_cast<int64_t>(T) * H * Dp;
  a.wp = a.wa + nchunks * H * (kChunk * kChunk);
  // warps per CTA: the CTAs of one head share nothing but the rows they read, so few warps spread over more SMs
  int nw = 4;
  while (nw > 1 && (cw * (nw / 2) >= E || static_cast<int64_t>(batch) * H * ceil_div(E, cw * nw) < device_sm_count())) nw /= 2;
  const size_t esz = dtype == B200_F32 ? 4 : 2;
  const size_t smem = 2 * sizeof(float) * (2 * kChunk * Dp + kChunk * kChunk + Dp + (kChunk * cw * nw * esz + 15) / 16 * 4);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 pgrid(ceil_div(max_len, kChunk), H, batch), sgrid(ceil_div(E, cw * nw), H, batch);
#define LAUNCH(TT, LPD)                                                                              \
  do {                                                                                               \
    {                                                                                                \
      ScopedKernelTimer timer("channel_prepare", st);                                                \
      launch_kernel(channel_prepare_kernel<TT, LPD / 4>, pgrid, dim3(128), 0, st, 1, 0, a);          \
      B200_CHECK_LAUNCH("channel_prepare_kernel");                                                   \
    }                                                                                                \
    auto kern = channel_scan_kernel<TT, LPD>;                                                        \
    if (smem > 48 * 1024)                                                                            \
      B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,           \
                                        static_cast<int>(smem)));                                    \
    ScopedKernelTimer timer("channel_scan", st);                                                     \
    launch_kernel(kern, sgrid, dim3(32 * nw), smem, st, 1, 0, a);                                    \
  } while (0)
#define BY_D(TT)                    \
  do {                              \
    if (lpd == 4) LAUNCH(TT, 4);    \
    else if (lpd == 8) LAUNCH(TT, 8); \
    else LAUNCH(TT, 16);            \
  } while (0)
  if (dtype == B200_BF16) BY_D(__nv_bfloat16);
  else if (dtype == B200_F16) BY_D(__half);
  else if (dtype == B200_F32) BY_D(float);
  else B200_REQUIRE(false, "b200_channel_chunks: dtype %d", dtype);
#undef BY_D
#undef LAUNCH
  note_variant("channel_chunks lanes%d warps%d", lpd, nw);
  B200_CHECK_LAUNCH("channel_scan_kernel");
  return 0;
}
