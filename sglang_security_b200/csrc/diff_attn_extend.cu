// Differential attention (see diff_attn.cu) of prompt portions on tcgen05 / TMEM for sm_100a.
//
// One CTA = (batch entry, key/value head, tile of 128 query rows); a row is a (token, query head) pair, PACK
// heads of one key/value head packed into the tile so that one gathered key/value tile feeds them all.
// BOTH maps of a row run in the same CTA: the query row [q1 | q2] and the key row [k1 | k2] are staged as
// stored, map m's scores are the product over its half of the coordinates, and both maps' weights meet the
// same value tile.  Keys and values therefore cross to shared memory once for two softmaxes, nothing is
// padded, and the difference, its norm and the 16-bit store happen in the epilogue from fp32 accumulators.
//
//   warps 0-3  : softmax of map 1 (thread = row): S1 tile TMEM -> registers, maximum, exp2, 16-bit weights to
//                swizzled shared memory, lazy rescale of O1
//   warps 4-7  : the same for map 2.  Epilogue: the two exchange halves of a_1 and lambda * a_2 through
//                shared memory (fp32), each finishes half of every row's columns
//   warp 8     : MMA issuer (one thread): S_m = Q_m K_m^T (M128 N64, K = D), O_m += P_m V (M128 N = DV, K64);
//                owns the TMEM allocation: S1 | S2 | O1 | O2
//   warps 9-11 : gather of 64-token key and value tiles through req_to_token (cp.async, 2 to 4 stages, up to
//                three tiles in flight)
// While one map's warps work on their tile the other map's products run, so the two maps hide each other.
// Every wait is bounded: a wait that runs out marks the host-visible error word and the CTA runs to its end
// without waiting further (all its addresses stay in bounds), so a fault is reported, not hung on.
#include <type_traits>

#include "tc_common.cuh"

namespace b200 {

struct DiffExtendParams {
  const void* q;               // [rows][H][2 * D]
  int64_t q_stride;
  const void* pool;
  int64_t kv_row_stride;
  int k_off, v_off;
  void* o;                     // [rows][H][DV]
  int64_t o_stride;
  const int32_t* req_to_token;
  int64_t rtt_stride;
  const int64_t* req_pool_indices;
  const int32_t *prefix_lens, *extend_lens, *extend_start;
  int group, pack, head_tiles;
  float qk_scale;              // scale * log2 e (> 0)
  int window, chunk;
  const float* lambda;
  float out_mult, eps;
  int* error;                  // host-mapped word: a bounded wait ran out
};

constexpr int kDxThreads = 384;
constexpr int kDxTile = 64;            // keys per tile
constexpr int kDxLoaders = 96;
constexpr float kDxRescale = 8.0f;     // log2 units
constexpr int kDxSpin = 1 << 24;       // limits of one wait: polls, and clock ticks (about a second)
constexpr long long kDxTicks = 2000000000ll;

template <int DK, int DV>
struct DiffExtendCfg {
  static constexpr int D = DK / 2;
  static constexpr int Q_BYTES = 128 * DK * 2, K_BYTES = kDxTile * DK * 2, V_BYTES = kDxTile * DV * 2;
  static constexpr int P_BYTES = 128 * kDxTile * 2;
  // as many key / value stages (2 to 4) as fit
  static constexpr int FREE = 226 * 1024 - Q_BYTES - 2 * P_BYTES;
  static constexpr int STAGES = FREE / (K_BYTES + V_BYTES) >= 4 ? 4 : FREE / (K_BYTES + V_BYTES);
  static_assert(STAGES >= 2, "two stages at least");
  static constexpr int OFF_Q = 0, OFF_K = Q_BYTES, OFF_V = OFF_K + STAGES * K_BYTES, OFF_P = OFF_V + STAGES * V_BYTES;
  static constexpr int OFF_BAR = OFF_P + 2 * P_BYTES;
  static constexpr int SMEM_BYTES = OFF_BAR + 256;
  static constexpr int S_COL = 0, O_COL = 2 * kDxTile;
  static constexpr int TMEM_COLS = O_COL + 2 * DV <= 256 ? 256 : 512;
  static_assert(O_COL + 2 * DV <= 512, "accumulators exceed tensor memory");
  static_assert(128 * DV * 4 <= OFF_P, "the epilogue's exchange buffer reuses the operand area");
  static_assert(SMEM_BYTES <= 227 * 1024, "tiles exceed shared memory");
};

template <int ROWS>
__device__ __forceinline__ uint32_t dx_swz(int row, int col) {
  return (col >> 3) * (ROWS * 128) + row * 128 + (((col & 7) ^ (row & 7)) << 4);
}

__device__ __forceinline__ float dx_max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;\n" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}

__device__ __forceinline__ int dx_first(int p, int window, int chunk) {
  return chunk > 0 ? p / chunk * chunk : (window > 0 ? max(0, p - window + 1) : 0);
}

template <typename T, int DK, int DV>
__global__ void __launch_bounds__(kDxThreads, 1)
diff_attn_extend_kernel(const DiffExtendParams p) {
  using C = DiffExtendCfg<DK, DV>;
  constexpr int D = C::D;
  extern __shared__ __align__(1024) uint8_t dx_smem[];
  const uint32_t sbase = smem_u32(dx_smem);
  const int warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;

  const int b = blockIdx.z, ext = p.extend_lens[b], prefix = p.prefix_lens[b];
  const int tok_per_tile = 128 / p.pack;
  // later rows see more keys (up to a chunk's edge): the last tiles are launched first
  const int tok0 = static_cast<int>(gridDim.x - 1 - blockIdx.x) * tok_per_tile;
  if (tok0 >= ext) return;             // uniform for the CTA
  if ((sbase & 1023u) != 0) {          // swizzled operands need a 1024-byte aligned base
    if (threadIdx.x == 0) *p.error = 2;
    return;
  }
  const int kvh = blockIdx.y / p.head_tiles;
  const int head_base = kvh * p.group + (blockIdx.y - kvh * p.head_tiles) * p.pack;
  const int kv_len = prefix + ext, tok_last = min(tok0 + tok_per_tile, ext) - 1;
  // key tiles from the first key that any row sees to the last one
  const int jb = dx_first(prefix + tok0, p.window, p.chunk) / kDxTile;
  const int n_kv = ceil_div(prefix + tok_last + 1, kDxTile) - jb;
  const int64_t q_row0 = p.extend_start[b];

  constexpr int ST = C::STAGES;
  const uint32_t bars = sbase + C::OFF_BAR, bar_q = bars;
  auto bar_s_full = [&](int m) { return bars + 8u * (1 + m); };
  auto bar_s_free = [&](int m) { return bars + 8u * (3 + m); };
  auto bar_p_full = [&](int m) { return bars + 8u * (5 + m); };
  auto bar_pv_full = [&](int m) { return bars + 8u * (7 + m); };
  auto bar_kv_full = [&](int s) { return bars + 8u * (9 + s); };
  auto bar_kv_empty = [&](int s) { return bars + 8u * (13 + s); };
  const uint32_t tmem_slot = bars + 8u * 17;
  volatile int* failed = reinterpret_cast<volatile int*>(dx_smem + C::OFF_BAR + 8 * 18);
  if (threadIdx.x == 0) {
    *failed = 0;
    tc::mbar_init(bar_q, kDxLoaders);
    for (int s = 0; s < ST; ++s) {
      tc::mbar_init(bar_kv_full(s), kDxLoaders);
      tc::mbar_init(bar_kv_empty(s), 1);
    }
    for (int s = 0; s < 2; ++s) {
      tc::mbar_init(bar_s_full(s), 1);
      tc::mbar_init(bar_s_free(s), 128);
      tc::mbar_init(bar_p_full(s), 128);
      tc::mbar_init(bar_pv_full(s), 1);
    }
    tc::fence_barrier_init();
  }
  if (warp == 8) {
    tc::tmem_alloc(tmem_slot, C::TMEM_COLS);
    tc::tmem_relinquish();
  }
  tc::tc_fence_before();
  __syncthreads();
  tc::tc_fence_after();
  const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(dx_smem + C::OFF_BAR + 8 * 17);
  auto wait = [&](uint32_t bar, uint32_t parity) {
    if (tc::mbar_try_wait(bar, parity)) return;
    const long long t0 = clock64();
    for (int i = 0; i < kDxSpin && clock64() - t0 < kDxTicks; ++i) {
      if (tc::mbar_try_wait(bar, parity)) return;
      if (*failed) return;
    }
    *failed = 1;
    *p.error = 1;
  };

  if (warp >= 9) {
    // ===================== gather loaders =====================
    const int lt = threadIdx.x - 9 * 32;
    const int32_t* rtt = p.req_to_token + p.req_pool_indices[b] * p.rtt_stride;
    const int64_t row_bytes = p.kv_row_stride * 2;
    const char* kbase = static_cast<const char*>(p.pool) + (static_cast<int64_t>(p.k_off) + kvh * DK) * 2;
    const char* vbase = static_cast<const char*>(p.pool) + (static_cast<int64_t>(p.v_off) + kvh * DV) * 2;
    constexpr int CK = DK / 8, CV = DV / 8;            // 16-byte pieces of a row
    for (int c = lt; c < 128 * CK; c += kDxLoaders) {  // row r = (token r / pack, head r % pack)
      const int r = c / CK, col = c - r * CK;
      int tok = tok0 + r / p.pack;
      if (tok >= ext) tok = ext - 1;                   // padding rows repeat the last token (never stored)
      const char* src = static_cast<const char*>(p.q) +
                        ((q_row0 + tok) * p.q_stride + static_cast<int64_t>(head_base + r % p.pack) * DK) * 2 + col * 16;
      cp_async16(sbase + C::OFF_Q + dx_swz<128>(r, col), src);
    }
    cp_async_commit();
    // a thread owns one 16-byte column of rows krow + KP * i of the keys, vrow + VP * i of the values; the
    // slots of tile j + 1 are fetched while tile j is in flight
    constexpr int KP = kDxLoaders / CK, KN = (kDxTile + KP - 1) / KP;
    constexpr int VP = kDxLoaders / CV, VN = (kDxTile + VP - 1) / VP;
    const int krow = lt / CK, kcol = lt - krow * CK, vrow = lt / CV, vcol = lt - vrow * CV;
    int32_t ks[KN], vs[VN];
    auto slot_of = [&](int j, int row) {
      const int pos = (jb + j) * kDxTile + row;
      return (row < kDxTile && pos < kv_len) ? __ldg(rtt + pos) : 0;     // 0 = the pool's dummy row
    };
    auto load_slots = [&](int j) {
#pragma unroll
      for (int i = 0; i < KN; ++i) ks[i] = slot_of(j, krow + KP * i);
      if constexpr (CK != CV) {
#pragma unroll
        for (int i = 0; i < VN; ++i) vs[i] = slot_of(j, vrow + VP * i);
      }
    };
    auto issue_tile = [&](int j) {
      const uint32_t sk = sbase + C::OFF_K + (j % ST) * C::K_BYTES, sv = sbase + C::OFF_V + (j % ST) * C::V_BYTES;
#pragma unroll
      for (int i = 0; i < KN; ++i) {
        const int r = krow + KP * i;
        if (r < kDxTile) cp_async16(sk + dx_swz<kDxTile>(r, kcol), kbase + ks[i] * row_bytes + kcol * 16);
      }
#pragma unroll
      for (int i = 0; i < VN; ++i) {
        const int r = vrow + VP * i;
        const int32_t sl = CK == CV ? ks[i < KN ? i : 0] : vs[i];
        if (r < kDxTile) cp_async16(sv + dx_swz<kDxTile>(r, vcol), vbase + sl * row_bytes + vcol * 16);
      }
      cp_async_commit();
    };
    // Tile j - LAG is published after tile j has been issued.  Before tile j may be issued, the product with
    // the values of tile j - ST must be done, and the issuer asks for tile j - ST + 1 = j - 1 - LAG first: it has
    // been published by then.
    constexpr int LAG = ST - 2;
    auto publish = [&](int j) {
      tc::fence_proxy_async_smem();
      if (j == 0) tc::mbar_arrive(bar_q);              // copied before tile 0
      tc::mbar_arrive(bar_kv_full(j % ST));
    };
    load_slots(0);
    for (int j = 0; j < n_kv; ++j) {
      if (j >= ST) wait(bar_kv_empty(j % ST), (j / ST - 1) & 1);
      issue_tile(j);
      if (j + 1 < n_kv) load_slots(j + 1);
      if (j >= LAG) {
        cp_async_wait<LAG>();
        publish(j - LAG);
      }
    }
    cp_async_wait<0>();
    for (int j = max(0, n_kv - LAG); j < n_kv; ++j) publish(j);
  } else if (warp == 8) {
    // ===================== MMA issuer =====================
    if (lane == 0) {
      constexpr uint32_t fmt = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;
      constexpr uint32_t idesc_qk = tc::make_idesc(fmt, fmt, 128, kDxTile, 0, 0);
      constexpr uint32_t idesc_pv = tc::make_idesc(fmt, fmt, 128, DV, 0, 1);   // V: MN-major B
      auto issue_qk = [&](int j, int m) {
        const uint32_t sk = sbase + C::OFF_K + (j % ST) * C::K_BYTES;
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk) {
          const int k = m * (D / 16) + kk;             // 16-coordinate step of the whole [map 1 | map 2] row
          const uint32_t qoff = (k >> 2) * (128 * 128) + (k & 3) * 32;
          const uint32_t koff = (k >> 2) * (kDxTile * 128) + (k & 3) * 32;
          tc::mma_f16(tmem_base + C::S_COL + m * kDxTile, tc::make_smem_desc_sw128(sbase + C::OFF_Q + qoff, 1024, 16),
                      tc::make_smem_desc_sw128(sk + koff, 1024, 16), idesc_qk, kk != 0 ? 1u : 0u);
        }
        tc::mma_commit(bar_s_full(m));
      };
      wait(bar_q, 0);
      wait(bar_kv_full(0), 0);
      tc::tc_fence_after();
      issue_qk(0, 0);
      issue_qk(0, 1);
      for (int j = 0; j < n_kv; ++j) {
        if (j + 1 < n_kv) {
          wait(bar_kv_full((j + 1) % ST), ((j + 1) / ST) & 1);
          for (int m = 0; m < 2; ++m) {
            wait(bar_s_free(m), j & 1u);               // the softmax has pulled S_m(j) out of TMEM
            tc::tc_fence_after();
            issue_qk(j + 1, m);
          }
        }
        const uint32_t sv = sbase + C::OFF_V + (j % ST) * C::V_BYTES;
        for (int m = 0; m < 2; ++m) {
          wait(bar_p_full(m), j & 1u);
          tc::tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < kDxTile / 16; ++kk)
            tc::mma_f16(tmem_base + C::O_COL + m * DV,
                        tc::make_smem_desc_sw128(sbase + C::OFF_P + m * C::P_BYTES + kk * 32, 1024, 16),
                        tc::make_smem_desc_sw128(sv + kk * 16 * 128, 1024, kDxTile * 128), idesc_pv,
                        (j | kk) != 0 ? 1u : 0u);
          tc::mma_commit(bar_pv_full(m));
        }
        tc::mma_commit(bar_kv_empty(j % ST));
      }
    }
  } else {
    // ===================== softmax (thread = query row of one map) =====================
    const int m_id = warp >> 2, r = (warp & 3) * 32 + lane;
    const int tok = tok0 + r / p.pack;
    const bool row_ok = tok < ext;
    const int limit = prefix + min(tok, ext - 1);                       // last visible key
    const int first = dx_first(limit, p.window, p.chunk);               // first visible key
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t tmem_s = tmem_base + lane_addr + C::S_COL + m_id * kDxTile;
    const uint32_t tmem_o = tmem_base + lane_addr + C::O_COL + m_id * DV;
    const uint32_t sp = sbase + C::OFF_P + m_id * C::P_BYTES;
    const float2 sc2 = make_float2(p.qk_scale, p.qk_scale), one2 = make_float2(1.f, 1.f);
    float m = -INFINITY, l = 0.f;
    for (int j = 0; j < n_kv; ++j) {
      wait(bar_s_full(m_id), j & 1u);
      tc::tc_fence_after();
      uint32_t v[2][32];
      tc::tmem_ld32(tmem_s, v[0]);
      tc::tmem_ld32(tmem_s + 32, v[1]);
      tc::tmem_ld_wait();
      tc::tc_fence_before();
      tc::mbar_arrive(bar_s_free(m_id));
      const int k0 = (jb + j) * kDxTile;
      if (k0 + kDxTile - 1 > limit || k0 < first) {
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            const int kp = k0 + h * 32 + c;
            if (kp > limit || kp < first) v[h][c] = 0xff800000u;        // -inf
          }
      }
      float a0 = -INFINITY, a1 = -INFINITY, a2 = -INFINITY, a3 = -INFINITY;
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int c = 0; c < 32; c += 8) {
          a0 = dx_max3(a0, __uint_as_float(v[h][c]), __uint_as_float(v[h][c + 1]));
          a1 = dx_max3(a1, __uint_as_float(v[h][c + 2]), __uint_as_float(v[h][c + 3]));
          a2 = dx_max3(a2, __uint_as_float(v[h][c + 4]), __uint_as_float(v[h][c + 5]));
          a3 = dx_max3(a3, __uint_as_float(v[h][c + 6]), __uint_as_float(v[h][c + 7]));
        }
      const float m_new = fmaxf(m, fmaxf(fmaxf(a0, a1), fmaxf(a2, a3)) * p.qk_scale);
      const bool need = m_new > m + kDxRescale;                         // also the first finite maximum
      bool pv_waited = false;
      if (__any_sync(0xffffffffu, need)) {
        if (j > 0) {
          wait(bar_pv_full(m_id), (j - 1) & 1u);                        // O_m holds tiles 0 .. j-1
          tc::tc_fence_after();
          pv_waited = true;
          const float alpha = (m == -INFINITY) ? 0.f : fast_exp2(m - m_new);
#pragma unroll 1
          for (int cc = 0; cc < DV / 32; ++cc) {
            uint32_t o[32];
            tc::tmem_ld32(tmem_o + cc * 32, o);
            tc::tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
            tc::tmem_st32(tmem_o + cc * 32, o);
          }
          tc::tmem_st_wait();
          l *= alpha;
        }
        m = m_new;
      }
      const float m_use = (m == -INFINITY) ? 0.f : m;
      uint32_t packed[2][16];
      const float2 nm2 = make_float2(-m_use, -m_use);
      float2 lsum = make_float2(0.f, 0.f);
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int c = 0; c < 16; ++c) {
          const float2 x = ffma2(make_float2(__uint_as_float(v[h][2 * c]), __uint_as_float(v[h][2 * c + 1])), sc2, nm2);
          const float p0 = fast_exp2(x.x), p1 = fast_exp2(x.y);
          lsum = ffma2(make_float2(p0, p1), one2, lsum);
          if constexpr (std::is_same<T, __nv_bfloat16>::value) {
            __nv_bfloat162 t2 = __floats2bfloat162_rn(p0, p1);
            packed[h][c] = *reinterpret_cast<uint32_t*>(&t2);
          } else {
            __half2 t2 = __floats2half2_rn(p0, p1);
            packed[h][c] = *reinterpret_cast<uint32_t*>(&t2);
          }
        }
      l += lsum.x + lsum.y;
      if (j > 0 && !pv_waited) {
        wait(bar_pv_full(m_id), (j - 1) & 1u);                          // P(j-1) has been read
        tc::tc_fence_after();
      }
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const uint32_t addr = sp + r * 128 + (((h * 4 + i) ^ (r & 7)) << 4);
          asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};\n" ::"r"(addr), "r"(packed[h][4 * i]),
                       "r"(packed[h][4 * i + 1]), "r"(packed[h][4 * i + 2]), "r"(packed[h][4 * i + 3])
                       : "memory");
        }
      tc::fence_proxy_async_smem();
      tc::tc_fence_before();
      tc::mbar_arrive(bar_p_full(m_id));
    }
    // ---- epilogue: the last products of BOTH maps must have read their operands before the exchange buffer
    //      (operand area, [column][row] fp32) is written: map 2's products are issued last and its commit
    //      covers everything before them.  The own map's barrier first: a parity wait is only unambiguous
    //      one phase ahead, and map 1's last product is issued after map 2's last but one
    wait(bar_pv_full(m_id), (n_kv - 1) & 1u);
    wait(bar_pv_full(1), (n_kv - 1) & 1u);
    tc::tc_fence_after();
    // map m's warps own half m of the columns: each hands its sums of the other half over
    constexpr int HC = DV / 2;
    const float f = (l > 0.f ? 1.0f / l : 0.f) * (m_id == 1 ? *p.lambda : 1.0f);
    float* give = reinterpret_cast<float*>(dx_smem) + m_id * HC * 128 + r;
    const float* take = reinterpret_cast<const float*>(dx_smem) + (1 - m_id) * HC * 128 + r;
    float* sums = reinterpret_cast<float*>(dx_smem + C::OFF_P) + r;     // [2][128], the weights are done with
#pragma unroll
    for (int cc = 0; cc < HC / 32; ++cc) {
      uint32_t o[32];
      tc::tmem_ld32(tmem_o + (1 - m_id) * HC + cc * 32, o);
      tc::tmem_ld_wait();
#pragma unroll
      for (int c = 0; c < 32; ++c) give[(cc * 32 + c) * 128] = __uint_as_float(o[c]) * f;
    }
    asm volatile("bar.sync 1, 256;\n" ::: "memory");
    float d[HC], ss = 0.f;
    const float own = m_id == 0 ? f : -f, other = m_id == 0 ? -1.0f : 1.0f;   // a_1 - lambda a_2 from either side
#pragma unroll
    for (int cc = 0; cc < HC / 32; ++cc) {
      uint32_t o[32];
      tc::tmem_ld32(tmem_o + m_id * HC + cc * 32, o);
      tc::tmem_ld_wait();
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        const float x = fmaf(__uint_as_float(o[c]), own, other * take[(cc * 32 + c) * 128]);
        ss = fmaf(x, x, ss);
        d[cc * 32 + c] = x;
      }
    }
    sums[m_id * 128] = ss;
    asm volatile("bar.sync 1, 256;\n" ::: "memory");
    const float mul = p.out_mult / sqrtf((sums[0] + sums[128]) * (1.0f / DV) + p.eps);
    if (row_ok) {
      T* orow = static_cast<T*>(p.o) + (q_row0 + tok) * p.o_stride +
                static_cast<int64_t>(head_base + r % p.pack) * DV + m_id * HC;
#pragma unroll
      for (int c8 = 0; c8 < HC / 8; ++c8) {
        alignas(16) T w[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = from_float<T>(d[c8 * 8 + e] * mul);
        *reinterpret_cast<uint4*>(orow + c8 * 8) = *reinterpret_cast<const uint4*>(w);
      }
    }
  }
  tc::tc_fence_before();
  __syncthreads();
  if (warp == 8) tc::tmem_dealloc(tmem_base, C::TMEM_COLS);
}

// One word of host memory that the device can write: set by a kernel whose bounded wait ran out.
static int* diff_error_word() {
  static int* word = [] {
    int* w = nullptr;
    if (cudaHostAlloc(reinterpret_cast<void**>(&w), sizeof(int), cudaHostAllocMapped) != cudaSuccess) {
      (void)cudaGetLastError();
      return static_cast<int*>(nullptr);
    }
    *w = 0;
    return w;
  }();
  return word;
}

template <typename T, int DK, int DV>
static int launch_diff_extend(const DiffExtendParams& p, int bs, int max_ext, int G, cudaStream_t st) {
  using C = DiffExtendCfg<DK, DV>;
  auto kern = diff_attn_extend_kernel<T, DK, DV>;
  static bool attr_done = false;
  if (!attr_done) {
    B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES));
    attr_done = true;
  }
  note_variant("diff_attn_extend dk=%d dv=%d pack=%d", DK, DV, p.pack);
  const dim3 grid(ceil_div(max_ext, 128 / p.pack), G * p.head_tiles, bs);
  {
    ScopedKernelTimer timer("diff_attn_extend", st);
    kern<<<grid, kDxThreads, C::SMEM_BYTES, st>>>(p);
  }
  B200_CHECK_LAUNCH("diff_attn_extend_kernel");
  return 0;
}

template <typename T>
static int dispatch_diff_extend(const DiffExtendParams& p, int D, int E, int bs, int max_ext, int G, cudaStream_t st) {
  const int dk = 2 * D;
#define CASE(K, V) if (dk == K && E == V) return launch_diff_extend<T, K, V>(p, bs, max_ext, G, st)
  CASE(64, 64); CASE(64, 128); CASE(128, 64); CASE(128, 128); CASE(256, 128);
#undef CASE
  B200_REQUIRE(false, "b200_diff_attn_extend: map size %d with value size %d", D, E);
}

}  // namespace b200

// 0, or the code a kernel left (1: a wait ran out); reading clears it
extern "C" int b200_diff_attn_extend_error(void) {
  int* w = b200::diff_error_word();
  if (!w) return 0;
  const int v = *static_cast<volatile int*>(w);
  *w = 0;
  return v;
}

extern "C" int b200_diff_attn_extend(const void* q, int64_t q_stride, const void* pool, int64_t ld_pool,
                                     int k_off, int v_off, void* o, int64_t o_stride,
                                     const int* req_to_token, int64_t rtt_stride,
                                     const int64_t* req_pool_indices, const int* prefix_lens,
                                     const int* extend_lens, const int* extend_start, int bs, int max_ext,
                                     int H, int G, int D, int E, float scale, int window, int chunk,
                                     const float* lambda, float out_mult, float eps, int dtype,
                                     void* stream) {
  using namespace b200;
  if (bs == 0 || max_ext == 0) return 0;
  B200_REQUIRE(q && pool && o && req_to_token && req_pool_indices && prefix_lens && extend_lens && extend_start && lambda,
               "b200_diff_attn_extend: null pointer");
  B200_REQUIRE(bs > 0 && bs <= 65535 && max_ext > 0 && H > 0 && G > 0 && H % G == 0 && scale > 0.f && window >= 0 &&
                   chunk >= 0 && !(window && chunk),
               "b200_diff_attn_extend: heads %d / %d, window %d, chunk %d", H, G, window, chunk);
  B200_REQUIRE(aligned16(q) && aligned16(pool) && aligned16(o) && q_stride % 8 == 0 && o_stride % 8 == 0 &&
                   ld_pool % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0,
               "b200_diff_attn_extend: rows must start on 16-byte boundaries");
  int* word = diff_error_word();
  B200_REQUIRE(word, "b200_diff_attn_extend: no host-visible error word");
  if (const int e = b200_diff_attn_extend_error())
    B200_REQUIRE(false, "b200_diff_attn_extend: an earlier launch gave up (code %d)", e);
  DiffExtendParams p;
  p.q = q;
  p.q_stride = q_stride;
  p.pool = pool;
  p.kv_row_stride = ld_pool;
  p.k_off = k_off;
  p.v_off = v_off;
  p.o = o;
  p.o_stride = o_stride;
  p.req_to_token = req_to_token;
  p.rtt_stride = rtt_stride;
  p.req_pool_indices = req_pool_indices;
  p.prefix_lens = prefix_lens;
  p.extend_lens = extend_lens;
  p.extend_start = extend_start;
  p.group = H / G;
  p.pack = 1;
  while (p.pack < 8 && p.group % (p.pack * 2) == 0) p.pack *= 2;   // largest power of two that divides the group
  p.head_tiles = p.group / p.pack;
  p.qk_scale = scale * 1.4426950408889634f;
  p.window = window;
  p.chunk = chunk;
  p.lambda = lambda;
  p.out_mult = out_mult;
  p.eps = eps;
  p.error = word;
  B200_REQUIRE(static_cast<int64_t>(G) * p.head_tiles <= 65535, "b200_diff_attn_extend: grid too large");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B200_BF16) return dispatch_diff_extend<__nv_bfloat16>(p, D, E, bs, max_ext, G, st);
  if (dtype == B200_F16) return dispatch_diff_extend<__half>(p, D, E, bs, max_ext, G, st);
  B200_REQUIRE(false, "b200_diff_attn_extend: dtype %d", dtype);
}
