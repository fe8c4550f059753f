// Differential attention over the paged one-row-per-token pool [keys | values]: every query head has two
// maps, q = [q1, q2] of size D each, every key/value head two key maps k = [k1, k2] and ONE value of size E;
//     a_m(i) = sum_j softmax_j(scale * q_m(i) . k_m(j)) v(j),   m = 1, 2
//     d = a_1 - lambda a_2;   o = d / sqrt(mean_e(d^2) + eps) * out_mult                (per query head)
// Position i sees the keys first(i) <= j <= i with first(i) = floor(i / chunk) * chunk (chunks counted from
// position 0), max(0, i - window + 1), or 0.
//
//   diff_attn     : CUDA cores, any size and dtype.  One CTA per (token, key/value head): both maps of two
//                   query heads per pass share the walk over the keys and every value row.  4 to 16 warps
//                   take tiles of 32 keys, each with a running maximum and sum per (head, map); merged in
//                   warp order; difference, norm and store in the same launch.  fp32 throughout.
//   diff_attn_mma : 16-bit pools, mma.sync m16n8k16, for decoded tokens and short portions.  The 16 rows of
//                   a tile are both maps of up to 8 query heads (rows 0-7 map 1, rows 8-15 map 2): with the
//                   key row [k1 | k2] as ONE operand of 2D coordinates and the query zero in the other map's
//                   half, one chain of products gives both maps' scores and one product with the value tile
//                   both maps' sums, so a key/value row is fetched once and no product is wasted.
//                   Split over the keys (grid.x); each warp streams its own ring of 16-token tiles with
//                   cp.async.  Scores, maxima and sums fp32, weights rounded for the product with the values.
//                   One split: difference and norm in the same launch; more: diff_attn_merge joins the parts.
#include <type_traits>

#include "common.cuh"

namespace b200 {

__device__ __forceinline__ int first_visible(int p, int window, int chunk) {
  return chunk > 0 ? p / chunk * chunk : (window > 0 ? max(0, p - window + 1) : 0);
}

struct DiffArgs {
  const void* q;               // [T, ldq]: per token [H][2][D] (fp32 for diff_attn, pool dtype for _mma)
  int64_t ldq;
  const void* pool;
  int64_t ld_pool;
  int k_off, v_off;
  const int* r2t;
  int64_t ld_r2t;
  const int64_t* req_idx;
  const int *tok_pos, *tok_b, *tok_list;
  const float* lambda;         // one number
  float out_mult, eps, scale;
  int window, chunk;
  void* out;                   // [T, ldo]: per token [H][E]
  int64_t ldo;
  int H, G, D, E;
  float *part_o, *part_lse;    // _mma with splits: [rows][H][2][splits]([E])
  int num_splits;
};

// ---- CUDA cores -------------------------------------------------------------------------------------
constexpr int kDiffMaxWarps = 16;
constexpr int kDiffMaxCols = 8;      // value size <= 256
constexpr int kDiffHeads = 2;        // query heads per pass (4 (head, map) rows)

template <typename TP, typename TO>
__global__ void __launch_bounds__(kDiffMaxWarps * 32)
diff_attn_kernel(const DiffArgs p) {
  extern __shared__ __align__(16) float da_smem[];
  constexpr int RH = kDiffHeads, NR = 2 * RH;
  const int nw = blockDim.x >> 5, D = p.D, E = p.E, R = p.H / p.G;
  const int Dp = (D + 3) & ~3;                 // rows of qs start on 16-byte boundaries
  float* qs = da_smem;                         // [NR][Dp] scaled queries: row 2 * head + map
  float* wacc = qs + NR * Dp;                  // [nw][NR][E]
  float* wm = wacc + nw * NR * E;              // [nw][NR]
  float* wl = wm + nw * NR;
  float* wf = wl + nw * NR;                    // merge factors
  float* wt = wf + nw * NR;                    // [NR] denominators
  const int t = p.tok_list ? p.tok_list[blockIdx.x] : blockIdx.x, g = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.tok_pos[t];
  const int* r2t = p.r2t + p.req_idx[p.tok_b[t]] * p.ld_r2t;
  const int lo = first_visible(pos, p.window, p.chunk), nkeys = pos - lo + 1;
  const TP* pool = static_cast<const TP*>(p.pool);
  const float* q = static_cast<const float*>(p.q) + t * p.ldq;
  TO* out = static_cast<TO*>(p.out) + t * p.ldo;
  const float lam = *p.lambda;
  constexpr int VK = 16 / sizeof(TP);          // elements of a 16-byte key load
  const bool vec = D % VK == 0 && p.ld_pool % VK == 0 && p.k_off % VK == 0 &&
                   (reinterpret_cast<uintptr_t>(pool) & 15) == 0;
  for (int h0 = 0; h0 < R; h0 += RH) {
    const int nh = min(RH, R - h0), hb = g * R + h0;
    __syncthreads();                           // the previous pass has finished with the shared arrays
    for (int i = threadIdx.x; i < NR * Dp; i += blockDim.x) {
      const int r = i / Dp, d = i - r * Dp;
      qs[i] = (r < 2 * nh && d < D) ? q[(hb * 2 + r) * D + d] * p.scale : 0.f;
    }
    __syncthreads();
    float m[NR], l[NR], acc[NR][kDiffMaxCols];
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      m[r] = -INFINITY;
      l[r] = 0.f;
#pragma unroll
      for (int c = 0; c < kDiffMaxCols; ++c) acc[r][c] = 0.f;
    }
    for (int n0 = warp * 32; n0 < nkeys; n0 += nw * 32) {
      const int n = n0 + lane;
      int64_t slot = 0;
      float s[NR];
#pragma unroll
      for (int r = 0; r < NR; ++r) s[r] = 0.f;
      if (n < nkeys) {
        slot = r2t[lo + n];
        const TP* kr = pool + slot * p.ld_pool + p.k_off + g * 2 * D;
#pragma unroll
        for (int map = 0; map < 2; ++map) {
          const TP* km = kr + map * D;
          if (vec) {
#pragma unroll 2
            for (int d = 0; d < D; d += VK) {
              const uint4 u = *reinterpret_cast<const uint4*>(km + d);
              const TP* e = reinterpret_cast<const TP*>(&u);
#pragma unroll
              for (int i = 0; i < VK; ++i) {
                const float kv = to_float<TP>(e[i]);
#pragma unroll
                for (int h = 0; h < RH; ++h)
                  s[2 * h + map] = fmaf(qs[(2 * h + map) * Dp + d + i], kv, s[2 * h + map]);
              }
            }
          } else {
            for (int d = 0; d < D; ++d) {
              const float kv = to_float<TP>(km[d]);
#pragma unroll
              for (int h = 0; h < RH; ++h)
                s[2 * h + map] = fmaf(qs[(2 * h + map) * Dp + d], kv, s[2 * h + map]);
            }
          }
        }
      }
      float pj[NR];
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const float sr = n < nkeys ? s[r] : -INFINITY;
        float tm = sr;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, o));
        const float mn = fmaxf(m[r], tm);
        const float corr = expf(m[r] - mn);    // first tile: exp(-inf) = 0
        pj[r] = n < nkeys ? expf(sr - mn) : 0.f;
        float ps = pj[r];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
        l[r] = l[r] * corr + ps;
        m[r] = mn;
#pragma unroll
        for (int c = 0; c < kDiffMaxCols; ++c) acc[r][c] *= corr;
      }
      const int cnt = min(32, nkeys - n0);
      for (int j0 = 0; j0 < cnt; j0 += 4) {    // the values of four keys in flight
#pragma unroll
        for (int c = 0; c < kDiffMaxCols; ++c) {
          if (32 * c >= E) continue;           // the same for all lanes
          const int e = lane + 32 * c;
          float x[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int64_t sl = __shfl_sync(0xffffffffu, slot, (j0 + i) & 31);   // lanes past cnt hold slot 0
            x[i] = e < E ? to_float<TP>(pool[sl * p.ld_pool + p.v_off + g * E + e]) : 0.f;
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) {
#pragma unroll
            for (int r = 0; r < NR; ++r) {
              const float pw = __shfl_sync(0xffffffffu, pj[r], (j0 + i) & 31);
              if (j0 + i < cnt) acc[r][c] = fmaf(pw, x[i], acc[r][c]);
            }
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      if (lane == 0) {
        wm[warp * NR + r] = m[r];
        wl[warp * NR + r] = l[r];
      }
#pragma unroll
      for (int c = 0; c < kDiffMaxCols; ++c) {
        const int e = lane + 32 * c;
        if (e < E) wacc[(warp * NR + r) * E + e] = acc[r][c];
      }
    }
    __syncthreads();
    if (threadIdx.x < NR) {
      const int r = threadIdx.x;
      float mt = -INFINITY;
      for (int w = 0; w < nw; ++w) mt = fmaxf(mt, wm[w * NR + r]);
      float lt = 0.f;
      for (int w = 0; w < nw; ++w) {
        const float f = wm[w * NR + r] == -INFINITY ? 0.f : expf(wm[w * NR + r] - mt);
        wf[w * NR + r] = f;
        lt = fmaf(wl[w * NR + r], f, lt);
      }
      wt[r] = lt;
    }
    __syncthreads();
    // one warp per head: the merged maps' difference stays in registers between the norm and the store
    for (int h = warp; h < nh; h += nw) {
      float d[kDiffMaxCols], ss = 0.f;
#pragma unroll
      for (int c = 0; c < kDiffMaxCols; ++c) {
        const int e = lane + 32 * c;
        d[c] = 0.f;
        if (e < E) {
          float o1 = 0.f, o2 = 0.f;
          for (int w = 0; w < nw; ++w) {
            o1 = fmaf(wacc[(w * NR + 2 * h) * E + e], wf[w * NR + 2 * h], o1);
            o2 = fmaf(wacc[(w * NR + 2 * h + 1) * E + e], wf[w * NR + 2 * h + 1], o2);
          }
          d[c] = o1 / wt[2 * h] - lam * (o2 / wt[2 * h + 1]);
          ss = fmaf(d[c], d[c], ss);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float r = p.out_mult / sqrtf(ss / static_cast<float>(E) + p.eps);
#pragma unroll
      for (int c = 0; c < kDiffMaxCols; ++c) {
        const int e = lane + 32 * c;
        if (e < E) out[(hb + h) * E + e] = from_float<TO>(d[c] * r);
      }
    }
  }
}

// ---- tensor cores, decoded tokens -----------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void diff_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                         uint32_t b0, uint32_t b1) {
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
        "{%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
  else
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
        "{%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void diff_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void diff_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
template <typename T>
__device__ __forceinline__ uint32_t diff_pack(float lo, float hi) {
  uint32_t r;
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;\n" : "=r"(r) : "f"(hi), "f"(lo));
  else
    asm("cvt.rn.f16x2.f32 %0, %1, %2;\n" : "=r"(r) : "f"(hi), "f"(lo));
  return r;
}

constexpr float kDiffLog2e = 1.4426950408889634f;
constexpr float kDiffNegBig = -1.0e30f;
constexpr int kDiffTile = 16;          // tokens per tile
constexpr int kDiffWarps = 4;
constexpr int kDiffAlign = kDiffTile * kDiffWarps;

// DK: both key maps of a head side by side (2 * D); DV: value size
template <int DK, int DV>
struct DiffMmaCfg {
  static constexpr int K_ROW = DK * 2, V_ROW = DV * 2;
  static constexpr int STAGE_BYTES = kDiffTile * (K_ROW + V_ROW);
  static constexpr int STAGES = STAGE_BYTES <= 6144 ? 4 : (STAGE_BYTES <= 8192 ? 3 : 2);
  static constexpr int RING_BYTES = kDiffWarps * STAGES * STAGE_BYTES;
  static constexpr int FINAL_BYTES = kDiffWarps * 16 * (DV + 2) * 4 + 16 * DV * 4;
  static constexpr int SMEM_BYTES = RING_BYTES > FINAL_BYTES ? RING_BYTES : FINAL_BYTES;
  static_assert(SMEM_BYTES <= 227 * 1024, "ring exceeds shared memory");
};

__host__ __device__ inline int diff_split_len(int len, int splits) {
  const int c = ceil_div(ceil_div(len, splits), kDiffAlign) * kDiffAlign;
  return c < kDiffAlign ? kDiffAlign : c;
}

template <typename T, int DK, int DV>
__global__ void __launch_bounds__(kDiffWarps * 32)
diff_attn_mma_kernel(const DiffArgs p) {
  using C = DiffMmaCfg<DK, DV>;
  constexpr int KS = DK / 16, NS = kDiffTile / 8, NO = DV / 8, STAGES = C::STAGES, D = DK / 2;
  extern __shared__ __align__(128) uint8_t dm_smem[];
  const int split = blockIdx.x, t = p.tok_list ? p.tok_list[blockIdx.z] : blockIdx.z;
  const int R = p.H / p.G, tiles = ceil_div(R, 8);
  const int g = blockIdx.y / tiles, h0 = (blockIdx.y - g * tiles) * 8, nh = min(8, R - h0);
  const int warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;
  const int pos = p.tok_pos[t], lo = first_visible(pos, p.window, p.chunk), len = pos - lo + 1;
  const int slen = diff_split_len(len, p.num_splits), s0 = split * slen;
  if (s0 >= len) return;
  const int start = lo + s0, end = min(pos + 1, start + slen);
  const int ntiles = ceil_div(end - start, kDiffTile);
  const int n_my = warp < ntiles ? (ntiles - warp + kDiffWarps - 1) / kDiffWarps : 0;
  const int* rtt = p.r2t + p.req_idx[p.tok_b[t]] * p.ld_r2t;

  // query fragments: map 1 lives in rows 0-7 and the first half of the coordinates, map 2 in rows 8-15 and
  // the second half; the other half of either is zero and never stored
  uint32_t qa[KS][2];
  {
    const int r = lane >> 2;
    const T* qb = static_cast<const T*>(p.q) + t * p.ldq + static_cast<int64_t>(g * R + h0 + r) * DK + (lane & 3) * 2;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      qa[ks][0] = r < nh ? *reinterpret_cast<const uint32_t*>(qb + ks * 16) : 0u;
      qa[ks][1] = r < nh ? *reinterpret_cast<const uint32_t*>(qb + ks * 16 + 8) : 0u;
    }
  }
  float o[NO][4];
#pragma unroll
  for (int i = 0; i < NO; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m1 = kDiffNegBig, m2 = kDiffNegBig, l1 = 0.f, l2 = 0.f;

  const char* kbase = static_cast<const char*>(p.pool) + (static_cast<int64_t>(p.k_off) + g * DK) * 2;
  const char* vbase = static_cast<const char*>(p.pool) + (static_cast<int64_t>(p.v_off) + g * DV) * 2;
  const int64_t row_bytes = p.ld_pool * 2;
  const uint32_t ring = smem_u32(dm_smem) + warp * (STAGES * C::STAGE_BYTES);
  int slot = 0;                         // lane & 15: the slot of that token of the next tile
  auto load_slots = [&](int k) {
    const int q = start + (warp + k * kDiffWarps) * kDiffTile + (lane & 15);
    slot = (k < n_my && q < end) ? __ldg(rtt + q) : 0;     // 0 = the pool's dummy row
  };
  auto issue_tile = [&](int k) {
    if (k < n_my) {                     // uniform for the warp
      const uint32_t sk = ring + (k % STAGES) * C::STAGE_BYTES, sv = sk + kDiffTile * C::K_ROW;
      constexpr int CK = DK / 8, CV = DV / 8;
#pragma unroll
      for (int i = 0; i < kDiffTile * CK / 32; ++i) {
        const int idx = lane + 32 * i, row = idx / CK, col = idx % CK;
        const int64_t sl = __shfl_sync(0xffffffffu, slot, row);
        cp_async16(sk + row * C::K_ROW + ((col ^ (row & 7)) << 4), kbase + sl * row_bytes + col * 16);
      }
#pragma unroll
      for (int i = 0; i < kDiffTile * CV / 32; ++i) {
        const int idx = lane + 32 * i, row = idx / CV, col = idx % CV;
        const int64_t sl = __shfl_sync(0xffffffffu, slot, row);
        cp_async16(sv + row * C::V_ROW + ((col ^ (row & 7)) << 4), vbase + sl * row_bytes + col * 16);
      }
    }
    cp_async_commit();
  };
  load_slots(0);
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    issue_tile(s);
    load_slots(s + 1);
  }
  const float mul = p.scale * kDiffLog2e;
  const int lx = lane & 7;
  const uint32_t k_row = lx * C::K_ROW, v_row = (((lane >> 3) & 1) * 8 + lx) * C::V_ROW;
  const int k_y = (lane >> 3) ^ lx, v_y = (lane >> 4) ^ lx;
  for (int it = 0; it < n_my; ++it) {
    issue_tile(it + STAGES - 1);
    load_slots(it + STAGES);
    cp_async_wait<STAGES - 1>();
    __syncwarp();
    const uint32_t sk = ring + (it % STAGES) * C::STAGE_BYTES, sv = sk + kDiffTile * C::K_ROW;
    const int tok0 = start + (warp + it * kDiffWarps) * kDiffTile;
    float s[NS][4];
#pragma unroll
    for (int nt = 0; nt < NS; ++nt) {
      s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ks += 2) {
        uint32_t kb[4];
        diff_ldsm(kb, sk + nt * 8 * C::K_ROW + k_row + (((2 * ks) ^ k_y) << 4));
        if (ks < KS / 2) {
          diff_mma<T>(s[nt], qa[ks][0], 0u, qa[ks][1], 0u, kb[0], kb[1]);
          if (KS > 2) diff_mma<T>(s[nt], qa[ks + 1][0], 0u, qa[ks + 1][1], 0u, kb[2], kb[3]);
          else diff_mma<T>(s[nt], 0u, qa[ks + 1][0], 0u, qa[ks + 1][1], kb[2], kb[3]);
        } else {
          diff_mma<T>(s[nt], 0u, qa[ks][0], 0u, qa[ks][1], kb[0], kb[1]);
          diff_mma<T>(s[nt], 0u, qa[ks + 1][0], 0u, qa[ks + 1][1], kb[2], kb[3]);
        }
      }
    }
    if (tok0 + kDiffTile > end) {
#pragma unroll
      for (int nt = 0; nt < NS; ++nt) {
        const int q = tok0 + nt * 8 + (lane & 3) * 2;
        if (q >= end) s[nt][0] = s[nt][2] = -INFINITY;
        if (q + 1 >= end) s[nt][1] = s[nt][3] = -INFINITY;
      }
    }
    float t1 = fmaxf(s[0][0], s[0][1]), t2 = fmaxf(s[0][2], s[0][3]);
#pragma unroll
    for (int nt = 1; nt < NS; ++nt) {
      t1 = fmaxf(t1, fmaxf(s[nt][0], s[nt][1]));
      t2 = fmaxf(t2, fmaxf(s[nt][2], s[nt][3]));
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, x));
      t2 = fmaxf(t2, __shfl_xor_sync(0xffffffffu, t2, x));
    }
    const float n1 = fmaxf(m1, t1 * mul), n2 = fmaxf(m2, t2 * mul);      // mul > 0 (host)
    if (__any_sync(0xffffffffu, n1 > m1 || n2 > m2)) {
      const float a1 = fast_exp2(m1 - n1), a2 = fast_exp2(m2 - n2);
      l1 *= a1;
      l2 *= a2;
#pragma unroll
      for (int i = 0; i < NO; ++i) {
        o[i][0] *= a1;
        o[i][1] *= a1;
        o[i][2] *= a2;
        o[i][3] *= a2;
      }
      m1 = n1;
      m2 = n2;
    }
    uint32_t pa[4];
#pragma unroll
    for (int nt = 0; nt < NS; ++nt) {
      const float p0 = fast_exp2(fmaf(s[nt][0], mul, -m1)), p1 = fast_exp2(fmaf(s[nt][1], mul, -m1));
      const float p2 = fast_exp2(fmaf(s[nt][2], mul, -m2)), p3 = fast_exp2(fmaf(s[nt][3], mul, -m2));
      l1 += p0 + p1;
      l2 += p2 + p3;
      pa[nt * 2] = diff_pack<T>(p0, p1);
      pa[nt * 2 + 1] = diff_pack<T>(p2, p3);
    }
#pragma unroll
    for (int np = 0; np < NO / 2; ++np) {
      uint32_t vb[4];
      diff_ldsm_t(vb, sv + v_row + (((2 * np) ^ v_y) << 4));
      diff_mma<T>(o[2 * np], pa[0], pa[1], pa[2], pa[3], vb[0], vb[1]);
      diff_mma<T>(o[2 * np + 1], pa[0], pa[1], pa[2], pa[3], vb[2], vb[3]);
    }
    __syncwarp();                       // the stage is refilled by the next iteration's issue
  }
  cp_async_wait<0>();
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    l1 += __shfl_xor_sync(0xffffffffu, l1, x);
    l2 += __shfl_xor_sync(0xffffffffu, l2, x);
  }
  __syncthreads();                      // every warp is done with its ring
  float* fin = reinterpret_cast<float*>(dm_smem);          // [warps][16][DV]
  float* fin_m = fin + kDiffWarps * 16 * DV;               // [warps][16]
  float* fin_l = fin_m + kDiffWarps * 16;
  float* res = fin_l + kDiffWarps * 16;                    // [16][DV] merged over the warps
  {
    const int r = lane >> 2, c0 = (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < NO; ++i) {
      *reinterpret_cast<float2*>(fin + (warp * 16 + r) * DV + i * 8 + c0) = make_float2(o[i][0], o[i][1]);
      *reinterpret_cast<float2*>(fin + (warp * 16 + r + 8) * DV + i * 8 + c0) = make_float2(o[i][2], o[i][3]);
    }
    if ((lane & 3) == 0) {
      fin_m[warp * 16 + r] = m1;
      fin_l[warp * 16 + r] = l1;
      fin_m[warp * 16 + r + 8] = m2;
      fin_l[warp * 16 + r + 8] = l2;
    }
  }
  __syncthreads();
  const int NSP = p.num_splits;
  for (int idx = threadIdx.x; idx < 16 * DV; idx += kDiffWarps * 32) {
    const int r = idx / DV, e = idx - r * DV, h = r & 7, map = r >> 3;
    if (h >= nh) continue;
    float M = fin_m[r];
#pragma unroll
    for (int w = 1; w < kDiffWarps; ++w) M = fmaxf(M, fin_m[w * 16 + r]);
    float num = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < kDiffWarps; ++w) {
      const float f = fast_exp2(fin_m[w * 16 + r] - M);    // idle warps: -1e30 -> 0
      num = fmaf(fin[(w * 16 + r) * DV + e], f, num);
      den = fmaf(fin_l[w * 16 + r], f, den);
    }
    const float val = num / den;
    if (NSP == 1) {
      res[r * DV + e] = val;
    } else {
      const int64_t i = ((static_cast<int64_t>(blockIdx.z) * p.H + g * R + h0 + h) * 2 + map) * NSP + split;
      p.part_o[i * DV + e] = val;
      if (e == 0) p.part_lse[i] = M + log2f(den);
    }
  }
  if (NSP > 1) return;
  __syncthreads();
  const float lam = *p.lambda;
  for (int h = warp; h < nh; h += kDiffWarps) {
    float d[DV / 32], ss = 0.f;
#pragma unroll
    for (int c = 0; c < DV / 32; ++c) {
      d[c] = res[h * DV + lane + 32 * c] - lam * res[(h + 8) * DV + lane + 32 * c];
      ss = fmaf(d[c], d[c], ss);
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float r = p.out_mult / sqrtf(ss / static_cast<float>(DV) + p.eps);
    T* out = static_cast<T*>(p.out) + t * p.ldo + static_cast<int64_t>(g * R + h0 + h) * DV;
#pragma unroll
    for (int c = 0; c < DV / 32; ++c) out[lane + 32 * c] = from_float<T>(d[c] * r);
  }
}

// The split parts of both maps joined, then difference, norm and store: one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(128)
diff_attn_merge_kernel(const DiffArgs p, int rows) {
  const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= rows * p.H) return;
  const int row = item / p.H, h = item - row * p.H, t = p.tok_list ? p.tok_list[row] : row;
  const int pos = p.tok_pos[t], len = pos - first_visible(pos, p.window, p.chunk) + 1;
  const int NSP = p.num_splits, nv = ceil_div(len, diff_split_len(len, NSP));
  const float lam = *p.lambda;
  float a[2][kDiffMaxCols];
#pragma unroll
  for (int map = 0; map < 2; ++map) {
    const int64_t base = (static_cast<int64_t>(item) * 2 + map) * NSP;
    float M = -INFINITY;
    for (int s = 0; s < nv; ++s) M = fmaxf(M, p.part_lse[base + s]);
    float den = 0.f;
#pragma unroll
    for (int c = 0; c < kDiffMaxCols; ++c) a[map][c] = 0.f;
    for (int s = 0; s < nv; ++s) {
      const float w = fast_exp2(p.part_lse[base + s] - M);
      den += w;
#pragma unroll
      for (int c = 0; c < kDiffMaxCols; ++c) {
        const int e = lane + 32 * c;
        if (e < p.E) a[map][c] = fmaf(w, p.part_o[(base + s) * p.E + e], a[map][c]);
      }
    }
    const float inv = 1.0f / den;
#pragma unroll
    for (int c = 0; c < kDiffMaxCols; ++c) a[map][c] *= inv;
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < kDiffMaxCols; ++c) {
    a[0][c] -= lam * a[1][c];
    ss = fmaf(a[0][c], a[0][c], ss);
  }
#pragma unroll
  for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
  const float r = p.out_mult / sqrtf(ss / static_cast<float>(p.E) + p.eps);
  T* out = static_cast<T*>(p.out) + t * p.ldo + static_cast<int64_t>(h) * p.E;
#pragma unroll
  for (int c = 0; c < kDiffMaxCols; ++c) {
    const int e = lane + 32 * c;
    if (e < p.E) out[e] = from_float<T>(a[0][c] * r);
  }
}

template <typename T, int DK, int DV>
static int launch_diff_mma_inst(const DiffArgs& p, int rows, cudaStream_t st) {
  using C = DiffMmaCfg<DK, DV>;
  auto kern = diff_attn_mma_kernel<T, DK, DV>;
  static bool attr_done = false;
  if (!attr_done) {
    B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES));
    attr_done = true;
  }
  note_variant("diff_attn_mma dk=%d dv=%d splits=%d", DK, DV, p.num_splits);
  const dim3 grid(p.num_splits, p.G * ceil_div(p.H / p.G, 8), rows);
  {
    ScopedKernelTimer timer("diff_attn_mma", st);
    B200_CUDA_OK(launch_kernel(kern, grid, dim3(kDiffWarps * 32), C::SMEM_BYTES, st, 1, 0, p));
  }
  B200_CHECK_LAUNCH("diff_attn_mma_kernel");
  if (p.num_splits > 1) {
    ScopedKernelTimer timer("diff_attn_merge", st);
    launch_kernel(diff_attn_merge_kernel<T>, dim3(ceil_div(rows * p.H, 4)), dim3(128), 0, st, 1, 0, p, rows);
    B200_CHECK_LAUNCH("diff_attn_merge_kernel");
  }
  return 0;
}

template <typename T>
static int launch_diff_mma(const DiffArgs& p, int rows, cudaStream_t st) {
  const int dk = 2 * p.D, dv = p.E;
#define CASE(K, V) if (dk == K && dv == V) return launch_diff_mma_inst<T, K, V>(p, rows, st)
  CASE(64, 64); CASE(64, 128); CASE(128, 64); CASE(128, 128); CASE(256, 128);
#undef CASE
  B200_REQUIRE(false, "b200_diff_attn_mma: map size %d with value size %d", p.D, p.E);
}

static int diff_check(const DiffArgs& p, int rows, const char* who) {
  B200_REQUIRE(p.q && p.pool && p.r2t && p.req_idx && p.tok_pos && p.tok_b && p.lambda && p.out, "%s: null pointer",
               who);
  B200_REQUIRE(rows > 0 && p.H > 0 && p.G > 0 && p.H % p.G == 0 && p.G <= 65535 && p.D > 0 && p.E > 0 &&
                   p.window >= 0 && p.chunk >= 0 && !(p.window && p.chunk) && p.E <= 32 * kDiffMaxCols,
               "%s: heads %d / %d, map size %d, value size %d (max %d), window %d, chunk %d", who, p.H, p.G, p.D,
               p.E, 32 * kDiffMaxCols, p.window, p.chunk);
  return 0;
}

}  // namespace b200

extern "C" int b200_diff_attn(const float* q, int64_t ldq, const void* pool, int64_t ld_pool, int k_off,
                              int v_off, const int* req_to_token, int64_t ld_r2t, const int64_t* req_idx,
                              const int* tok_pos, const int* tok_b, const int* tok_list,
                              const float* lambda, float out_mult, float eps, float scale, int window,
                              int chunk, void* out, int64_t ldo, int rows, int H, int G, int D, int E,
                              int max_keys, int dtype, void* stream) {
  using namespace b200;
  if (rows == 0) return 0;
  DiffArgs p{q, ldq, pool, ld_pool, k_off, v_off, req_to_token, ld_r2t, req_idx, tok_pos, tok_b, tok_list, lambda,
             out_mult, eps, scale, window, chunk, out, ldo, H, G, D, E, nullptr, nullptr, 1};
  if (int rc = diff_check(p, rows, "b200_diff_attn")) return rc;
  int nw = max_keys <= 0 ? 4 : min(kDiffMaxWarps, max(4, ceil_div(max_keys, 64)));
  auto smem_for = [&](int w) {
    return sizeof(float) * (2 * kDiffHeads * (static_cast<size_t>((D + 3) & ~3) + static_cast<size_t>(w) * (E + 3) + 1));
  };
  while (nw > 1 && smem_for(nw) > 48 * 1024) nw >>= 1;
  B200_REQUIRE(smem_for(nw) <= 48 * 1024, "b200_diff_attn: map size %d too large", D);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  note_variant("diff_attn warps=%d", nw);
  ScopedKernelTimer timer("diff_attn", st);
#define LAUNCH(TT) \
  launch_kernel(diff_attn_kernel<TT, TT>, dim3(rows, G), dim3(nw * 32), smem_for(nw), st, 1, 0, p)
  if (dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half);
  else if (dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_diff_attn: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("diff_attn_kernel");
  return 0;
}

extern "C" int b200_diff_attn_mma_supported(int D, int E) {
  const int dk = 2 * D;
  return (dk == 64 && (E == 64 || E == 128)) || (dk == 128 && (E == 64 || E == 128)) || (dk == 256 && E == 128);
}

// As many splits as keep all CTAs resident at once (two per SM: a second, partly filled wave costs more than
// longer parts), never fewer than 4 tiles of work per warp and part
extern "C" int b200_diff_attn_mma_splits(int rows, int H, int G, int max_keys, int num_sms) {
  using namespace b200;
  if (rows <= 0 || G <= 0 || H <= 0 || max_keys <= 0) return 1;
  const int64_t base = static_cast<int64_t>(rows) * G * ceil_div(H / G, 8);
  int64_t s = 2 * static_cast<int64_t>(num_sms) / base;
  const int64_t most = ceil_div(max_keys, 4 * kDiffAlign);
  s = s < most ? s : most;
  return static_cast<int>(s < 1 ? 1 : (s > 64 ? 64 : s));
}

extern "C" int b200_diff_attn_mma(const void* q, int64_t ldq, const void* pool, int64_t ld_pool, int k_off,
                                  int v_off, const int* req_to_token, int64_t ld_r2t,
                                  const int64_t* req_idx, const int* tok_pos, const int* tok_b,
                                  const int* tok_list, const float* lambda, float out_mult, float eps,
                                  float scale, int window, int chunk, void* out, int64_t ldo, int rows,
                                  int H, int G, int D, int E, int num_splits, float* part_o,
                                  float* part_lse, int dtype, void* stream) {
  using namespace b200;
  if (rows == 0) return 0;
  DiffArgs p{q, ldq, pool, ld_pool, k_off, v_off, req_to_token, ld_r2t, req_idx, tok_pos, tok_b, tok_list, lambda,
             out_mult, eps, scale, window, chunk, out, ldo, H, G, D, E, part_o, part_lse, num_splits};
  if (int rc = diff_check(p, rows, "b200_diff_attn_mma")) return rc;
  B200_REQUIRE(b200_diff_attn_mma_supported(D, E) && scale > 0.f, "b200_diff_attn_mma: map size %d, value size %d", D, E);
  B200_REQUIRE(num_splits >= 1 && num_splits <= 1024 && (num_splits == 1 || (part_o && part_lse)) && rows <= 65535,
               "b200_diff_attn_mma: %d splits of %d rows", num_splits, rows);
  B200_REQUIRE(aligned16(pool) && ld_pool % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 && ldq % 2 == 0 &&
                   (reinterpret_cast<uintptr_t>(q) & 3) == 0,
               "b200_diff_attn_mma: pool rows must start on 16-byte boundaries");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B200_BF16) return launch_diff_mma<__nv_bfloat16>(p, rows, st);
  if (dtype == B200_F16) return launch_diff_mma<__half>(p, rows, st);
  B200_REQUIRE(false, "b200_diff_attn_mma: dtype %d", dtype);
}
