// The channel-gated memory of linear_recurrence.cu (S <- diag(f) S + w v^T, w = 1 - f, then o = S^T q) for long
// prompt portions, 16 tokens at a time.  Within a chunk that starts from S_0, with f_(a,b] = prod_{a < s <= b} f_s
// per channel:
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
//   channel_scan    : one warp owns XC * 32 / (D / 8) value columns of a head for the whole portion; a lane holds
//                     8 channels x XC columns (2 or 4) of S in registers, channel pairs packed.  Per chunk: the 16 x XC
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
  float* work;                 // [chunk][H] blocks of q [16][Dp], k [16][Dp], A [16 j][16 i], decay [Dp]
  float* out;
  int64_t ldo;
  int H, D, E;
};

// chunk number c of batch entry b: ids of different entries do not meet, and stay below T / 16 + batch + 1
__device__ __forceinline__ int64_t chunk_id(int start, int b, int c) { return start / kChunk + b + c; }

__host__ __device__ constexpr int chunk_block(int Dp) { return 2 * kChunk * Dp + kChunk * kChunk + Dp; }

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
__global__ void __launch_bounds__(128, CPL == 4 ? 3 : 4)
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
  auto put = [&](float* dst, const float (&x)[CPL]) {
    if constexpr (CPL == 4) *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
    else if constexpr (CPL == 2) *reinterpret_cast<float2*>(dst) = make_float2(x[0], x[1]);
    else dst[0] = x[0];
  };
  // the warp's tokens: all loads requested before the first use, a lane's channels in one access where the
  // rows allow it
  struct __align__(sizeof(T) * CPL) Row { T x[CPL]; };
  const bool vec = a.D % CPL == 0 && a.ldq % CPL == 0 && a.ldf % CPL == 0 &&
                   reinterpret_cast<uintptr_t>(a.q) % sizeof(Row) == 0 && reinterpret_cast<uintptr_t>(a.zf) % sizeof(Row) == 0;
  Row qr[kChunk / 4], zr[kChunk / 4];
#pragma unroll
  for (int k = 0; k < kChunk / 4; ++k) {
    const int i = warp + 4 * k;
#pragma unroll
    for (int c = 0; c < CPL; ++c) qr[k].x[c] = zr[k].x[c] = from_float<T>(0.f);
    if (i >= n) continue;
    if (vec) {
      if (d0 < a.D) {
        qr[k] = *reinterpret_cast<const Row*>(qg + (row0 + i) * a.ldq);
        zr[k] = *reinterpret_cast<const Row*>(zg + (row0 + i) * a.ldf);
      }
    } else {
#pragma unroll
      for (int c = 0; c < CPL; ++c)
        if (d0 + c < a.D) {
          qr[k].x[c] = qg[(row0 + i) * a.ldq + c];
          zr[k].x[c] = zg[(row0 + i) * a.ldf + c];
        }
    }
  }
#pragma unroll
  for (int k = 0; k < kChunk / 4; ++k) {
    const int i = warp + 4 * k;
    float y[CPL], w[CPL];
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const bool in = i < n && d0 + c < a.D;
      const float q = to_float<T>(qr[k].x[c]);
      y[c] = (a.act == 1 ? __fdividef(q, 1.0f + expf(-q)) : q) * a.q_scale;
      w[c] = in ? __fdividef(1.0f - lo[c], 1.0f + expf(to_float<T>(zr[k].x[c]) + bi[c])) : 0.f;   // the written share
    }
    put(&qs[i][d0], y);
    put(&ws[i][d0], w);
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
  float* blk = a.work + (cid * a.H + h) * chunk_block(Dp);
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
    if ((i & 3) == warp) put(blk + i * Dp + d0, y);
  }
  if (warp == 0) put(blk + 2 * kChunk * Dp + kChunk * kChunk + d0, p);
#pragma unroll
  for (int c = 0; c < CPL; ++c) p[c] = 1.f;
#pragma unroll
  for (int j = kChunk - 1; j >= 0; --j) {
    if ((j & 3) == warp) {
      float y[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) y[c] = ws[j][d0 + c] * p[c];
      put(blk + (kChunk + j) * Dp + d0, y);
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c) p[c] *= f[j][c];
  }
  float* A = blk + 2 * kChunk * Dp;
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
    // the 16-byte pieces of row j are stored in the order (piece ^ j / 2 % 4): lanes that read one piece of 8
    // rows out of shared memory meet no bank twice
    if (!(lane & 1)) A[j * kChunk + ((lane >> 1) ^ (((j >> 1) & 3) << 2))] = part[0];
  }
}

// LPD lanes share a column group: Dp = 8 * LPD channels, XC (2 or 4) columns
template <typename T, int LPD, int XC>
__global__ void __launch_bounds__(128)
channel_scan_kernel(const ChunkArgs a) {
  constexpr int Dp = 8 * LPD, CW = XC * (32 / LPD), JL = kChunk / LPD;   // columns per warp; rows i, j per lane
  extern __shared__ __align__(16) float cs_smem[];
  const int b = blockIdx.z, h = blockIdx.y, len = a.ext_len[b];
  if (len < a.min_len) return;
  const int NT = blockDim.x, ES = (NT >> 5) * CW, e0 = blockIdx.x * ES;
  const int start = a.ext_start[b], E = a.E, H = a.H;
  const bool fresh = a.tok_pos[start] == 0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane % LPD, cl = warp * CW + (lane / LPD) * XC, e = e0 + cl;
  // one stage: the prepared block, v [16][ES] (in T, padded to 16 bytes)
  constexpr int v_at = chunk_block(Dp);
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
    const float* src = a.work + (cid * H + h) * chunk_block(Dp);
#pragma unroll 4
    for (int x = tid; x < chunk_block(Dp) / 4; x += NT) cp_async16(smem_u32(buf + 4 * x), src + 4 * x);
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
  f32x2 s[2][2][XC];                           // [atom][row pair][column]
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int c2 = 0; c2 < XC / 2; ++c2) {
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
  const bool out_vec = E % XC == 0 && a.ldo % XC == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
  const int chunks = (len + kChunk - 1) / kChunk;
  struct __align__(sizeof(T) * XC) Cols { T x[XC]; };
  auto values = [&](const T* vs, int j, float (&x)[XC]) {     // this lane's columns of row j
    const Cols u = *reinterpret_cast<const Cols*>(vs + j * ES + cl);
#pragma unroll
    for (int c = 0; c < XC; ++c) x[c] = to_float<T>(u.x[c]);
  };
  stage(0, cs_smem);
  for (int c = 0; c < chunks; ++c) {
    cp_async_wait<0>();
    __syncthreads();                           // chunk c is in; every warp has left chunk c - 1
    if (c + 1 < chunks) stage(c + 1, cs_smem + ((c + 1) & 1) * stage_floats);
    const float* buf = cs_smem + (c & 1) * stage_floats;
    const float *qs = buf, *ks = buf + kChunk * Dp, *As = ks + kChunk * Dp, *ps = As + kChunk * kChunk;
    const T* vs = reinterpret_cast<const T*>(buf + v_at);
    float vl[JL][XC];                          // the rows j this lane contributes to the inner sums
#pragma unroll
    for (int k = 0; k < JL; ++k) values(vs, g + k * LPD, vl[k]);
    float part[kChunk * XC];
#pragma unroll
    for (int ig = 0; ig < kChunk / 4; ++ig) {
      f32x2 acc[4][XC];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const ulonglong2 q0 = *reinterpret_cast<const ulonglong2*>(qs + (4 * ig + i) * Dp + 4 * g);
        const ulonglong2 q1 = *reinterpret_cast<const ulonglong2*>(qs + (4 * ig + i) * Dp + 4 * (LPD + g));
#pragma unroll
        for (int x = 0; x < XC; ++x) {
          acc[i][x] = mul2(s[0][0][x], q0.x);
          acc[i][x] = fma2(s[0][1][x], q0.y, acc[i][x]);
          acc[i][x] = fma2(s[1][0][x], q1.x, acc[i][x]);
          acc[i][x] = fma2(s[1][1][x], q1.y, acc[i][x]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int x = 0; x < XC; ++x) {
          float lo, hi;
          unpack2(acc[i][x], lo, hi);
          part[(4 * ig + i) * XC + x] = lo + hi;
        }
#pragma unroll
      for (int k = 0; k < JL; ++k) {
        const int j = g + k * LPD;
        const float4 A4 = *reinterpret_cast<const float4*>(As + j * kChunk + 4 * (ig ^ ((j >> 1) & 3)));
        const float Ai[4] = {A4.x, A4.y, A4.z, A4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int x = 0; x < XC; ++x) part[(4 * ig + i) * XC + x] = fmaf(Ai[i], vl[k][x], part[(4 * ig + i) * XC + x]);
      }
    }
    // sum over the LPD lanes of a column group; the lane keeps rows g * JL ... g * JL + JL - 1
    if constexpr (LPD == 16) {
      halve<8 * XC>(part, 8, g & 8);
      halve<4 * XC>(part, 4, g & 4);
      halve<2 * XC>(part, 2, g & 2);
      halve<XC>(part, 1, g & 1);
    } else if constexpr (LPD == 8) {
      halve<8 * XC>(part, 4, g & 4);
      halve<4 * XC>(part, 2, g & 2);
      halve<2 * XC>(part, 1, g & 1);
    } else {
      halve<8 * XC>(part, 2, g & 2);
      halve<4 * XC>(part, 1, g & 1);
    }
    const int n = min(kChunk, len - c * kChunk);
#pragma unroll
    for (int r = 0; r < JL; ++r) {
      const int i = g * JL + r;
      if (i < n && e < E) {
        float* dst = a.out + (start + c * kChunk + i) * a.ldo + h * E + e;
        if (out_vec) {
          if constexpr (XC == 4)
            *reinterpret_cast<float4*>(dst) = make_float4(part[r * 4], part[r * 4 + 1], part[r * 4 + 2], part[r * 4 + 3]);
          else
            *reinterpret_cast<float2*>(dst) = make_float2(part[r * 2], part[r * 2 + 1]);
        } else {
#pragma unroll
          for (int x = 0; x < XC; ++x)
            if (e + x < E) dst[x] = part[r * XC + x];
        }
      }
    }
    // S <- diag(decay) S + sum_j k_j v_j^T
    {
      const ulonglong2 p0 = *reinterpret_cast<const ulonglong2*>(ps + 4 * g);
      const ulonglong2 p1 = *reinterpret_cast<const ulonglong2*>(ps + 4 * (LPD + g));
#pragma unroll
      for (int x = 0; x < XC; ++x) {
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
      float xv[XC];
      values(vs, j, xv);
#pragma unroll
      for (int x = 0; x < XC; ++x) {
        const f32x2 vv = pack2(xv[x], xv[x]);
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
    for (int c2 = 0; c2 < XC / 2; ++c2) {
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
  return (static_cast<int64_t>(T) / kChunk + batch + 1) * H * chunk_block(8 * chunk_lanes(D));
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
  const int lpd = chunk_lanes(D), Dp = 8 * lpd;
  // 4 columns per lane, or 2 where that leaves schedulers without a warp (measured at 32 heads of 64 x 128: 186
  // against 249 us, at 64 heads of 128 x 128: 443 against 349 us)
  const int xc = static_cast<int64_t>(batch) * H * ceil_div(E, 4 * (32 / lpd)) < 4 * device_sm_count() ? 2 : 4;
  const int cw = xc * (32 / lpd);
  ChunkArgs a{q, zf, v, ldq, ldf, ldv, f_bias, f_lower, q_scale, act, min_len, state, ld_state, slot, tok_pos, ext_start,
              ext_len, work, out, ldo, H, D, E};
  // warps per CTA share the staged rows; fewer where that fills more SMs
  int nw = 4;
  while (nw > 1 && (cw * (nw / 2) >= E || static_cast<int64_t>(batch) * H * ceil_div(E, cw * nw) < device_sm_count())) nw /= 2;
  const size_t esz = dtype == B200_F32 ? 4 : 2;
  const size_t smem = 2 * sizeof(float) * (chunk_block(Dp) + (kChunk * cw * nw * esz + 15) / 16 * 4);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 pgrid(ceil_div(max_len, kChunk), H, batch), sgrid(ceil_div(E, cw * nw), H, batch);
#define LAUNCH(TT, LPD)                                                                              \
  do {                                                                                               \
    {                                                                                                \
      ScopedKernelTimer timer("channel_prepare", st);                                                \
      launch_kernel(channel_prepare_kernel<TT, LPD / 4>, pgrid, dim3(128), 0, st, 1, 0, a);          \
      B200_CHECK_LAUNCH("channel_prepare_kernel");                                                   \
    }                                                                                                \
    auto kern = xc == 4 ? channel_scan_kernel<TT, LPD, 4> : channel_scan_kernel<TT, LPD, 2>;                                                       \
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
  note_variant("channel_chunks lanes%d columns%d warps%d", lpd, xc, nw);
  B200_CHECK_LAUNCH("channel_scan_kernel");
  return 0;
}
