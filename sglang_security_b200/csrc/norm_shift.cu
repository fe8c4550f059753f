// Row kernels around a 32-bit residual stream, for model designs that keep the residual, the norms
// and the previous-token mix in fp32 while the matrix products run in the model dtype:
//   scalar_rmsnorm_shift : h = x / sqrt(mean(x^2) + eps) * gain (* weight[d]), and optionally the
//                          token-shifted copy hm = h + (h_prev - h) * mu[d], where h_prev is the h of
//                          the previous token of the same sequence: the row before it in this batch,
//                          the per-sequence state row if the token opens its portion, zeros at
//                          position 0.  The state row is replaced by the h of the portion's last token.
//   residual_combine     : x += a + b + sum_k w[t,k] * y[t*top+k] + g[t] * s[t]   (all terms optional)
//   act_and_mul          : out = act(z[:, :d]) * z[:, d:]  with act = silu or the tanh form of gelu
//   add_normed           : for designs whose norm sits on a sublayer's OUTPUT: y = sa * a + sb * b +
//                          sum_k rows[t * top + k] (all terms optional) in fp32, then
//                          x += mult * y / sqrt(mean(y^2) + eps) * w[d]; optionally also writes the new x
//                          in the model dtype, the next sublayer's input; with a second weight the copy is
//                          the NEXT sublayer's pre-norm instead, x / sqrt(mean(x^2) + eps) * w_next (designs
//                          with a norm on both sides of every sublayer: one launch per sublayer boundary)
//   add_normed_mix       : add_normed with every term a mixture-of-experts sublayer and a looped stack need:
//                          y = sa * a + sb * gb[t] * b + sum_k wts[t, k] * (ids[t, k] < n_experts ?
//                          rows[t * top + k] : same[t]) — a per-token gate on b, weighted expert rows, identity
//                          experts that return their input —, then x as above, then x += table[id_t] (a row of
//                          an embedding table, ahead of the next pass of a loop), then the copy / pre-norm.  16-byte
//                          loads, y and x stay in registers between the two norms (wide or unaligned rows: in shared
//                          memory).
//   softcap_rows         : out = cap * tanh(z / cap) in fp32
//   scaled_add_layernorm : for designs whose norm sits AFTER the residual sum: y = alpha * x + a + b +
//                          sum_k wts[t, k] * rows[t * top + k] (terms optional) in fp32, then
//                          x = (y - mean) / sqrt(var + eps) * w + bias (two passes: the variance is the
//                          mean of the squared deviations); optionally the copy of the new x in the
//                          model dtype.  With `in_place` = 0 x is left alone and only the copy is
//                          written (a model's final layer norm).
//   act_and_mul_clamped  : out = g * sigmoid(slope * g) * (u + 1), g = min(z[:, :d], limit),
//                          u = clamp(z[:, d:], -limit, limit)
//   xielu_rows           : out = xielu(z; pos, neg) (activation.cuh); the result may be a column slice of
//                          wider rows
#include "activation.cuh"
#include "common.cuh"

namespace b200 {

constexpr int kRowThreads = 256;

__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();  // red may still be read from the previous call
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = (l < kRowThreads / 32) ? red[l] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  return t;
}

__device__ __forceinline__ float row_inv_rms(const float* row, int W, float eps, float* red) {
  float s = 0.f;
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    const float v = row[d];
    s = fmaf(v, v, s);
  }
  s = block_sum(s, red);
  return 1.0f / sqrtf(s / static_cast<float>(W) + eps);
}

template <typename TO>
__global__ void __launch_bounds__(kRowThreads)
scalar_rmsnorm_shift_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ gain,
                            const float* __restrict__ weight, float eps,
                            const float* __restrict__ mu, float* __restrict__ state, int64_t ld_state,
                            const int* __restrict__ tok_pos, const int* __restrict__ tok_b,
                            const int* __restrict__ ext_start, const int* __restrict__ ext_len,
                            const int64_t* __restrict__ slot, TO* __restrict__ out_h, int64_t ldh,
                            TO* __restrict__ out_hm, int64_t ldm, int W) {
  __shared__ float red[kRowThreads / 32];
  const int t = blockIdx.x;
  const float g = gain ? *gain : 1.0f;
  const float* row = x + t * ldx;
  const float r = row_inv_rms(row, W, eps, red) ;
  if (!mu) {
    for (int d = threadIdx.x; d < W; d += kRowThreads) {
      float h = row[d] * r * g;
      if (weight) h *= weight[d];
      out_h[t * ldh + d] = from_float<TO>(h);
    }
    return;
  }
  const int b = tok_b[t];
  const int start = ext_start[b];
  const bool first = (t == start);
  const int pos = tok_pos[t];
  // 0: zeros, 1: the state row, 2: the previous row of this batch
  const int src = pos == 0 ? 0 : (first ? 1 : 2);
  float rp = 0.f;
  const float* prow = row - ldx;
  if (src == 2) rp = row_inv_rms(prow, W, eps, red);
  const int last = start + ext_len[b] - 1;
  float* srow = state ? state + slot[b] * ld_state : nullptr;
  float rl = r;
  const float* lrow = x + last * ldx;
  if (first && srow && last != t) rl = row_inv_rms(lrow, W, eps, red);
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    const float wd = weight ? weight[d] * g : g;
    const float h = row[d] * r * wd;
    float hp = 0.f;
    if (src == 1) hp = srow[d];
    else if (src == 2) hp = prow[d] * rp * wd;
    if (out_h) out_h[t * ldh + d] = from_float<TO>(h);
    out_hm[t * ldm + d] = from_float<TO>(h + (hp - h) * mu[d]);
    if (first && srow) srow[d] = (last == t) ? h : lrow[d] * rl * wd;   // same thread read srow[d] above
  }
}

template <typename TA>
__global__ void __launch_bounds__(kRowThreads)
residual_combine_kernel(float* __restrict__ x, int64_t ldx, const TA* __restrict__ a, int64_t lda,
                        const TA* __restrict__ b, int64_t ldb, const TA* __restrict__ y, int64_t ldy,
                        const float* __restrict__ topk_w, int top, const TA* __restrict__ s,
                        int64_t lds, const float* __restrict__ gate, int W) {
  const int t = blockIdx.x;
  const float g = gate ? gate[t] : 1.0f;
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    float acc = 0.f;
    if (a) acc += to_float<TA>(a[t * lda + d]);
    if (b) acc += to_float<TA>(b[t * ldb + d]);
    if (y) {
      float m = 0.f;
      for (int k = 0; k < top; ++k)
        m = fmaf(topk_w[t * top + k], to_float<TA>(y[(static_cast<int64_t>(t) * top + k) * ldy + d]), m);
      acc += m;
    }
    if (s) acc = fmaf(g, to_float<TA>(s[t * lds + d]), acc);
    x[t * ldx + d] += acc;
  }
}

__device__ __forceinline__ float act_apply(float z, int kind) {
  if (kind == 0) return z / (1.0f + expf(-z));                      // silu
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);  // gelu, tanh form
  return 0.5f * z * (1.0f + tanhf(u));
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
act_and_mul_kernel(const T* __restrict__ z, int64_t ldz, T* __restrict__ out, int64_t ldo, int D,
                   int kind) {
  const int t = blockIdx.x;
  for (int d = threadIdx.x; d < D; d += kRowThreads) {
    // the activation's value is rounded to the storage type before the product, as a chain of
    // separate operators would round it
    const float a = to_float<T>(from_float<T>(act_apply(to_float<T>(z[t * ldz + d]), kind)));
    out[t * ldo + d] = from_float<T>(a * to_float<T>(z[t * ldz + D + d]));
  }
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
xielu_rows_kernel(const T* __restrict__ z, int64_t ldz, T* __restrict__ out, int64_t ldo, int D, float pos,
                  float neg) {
  const int t = blockIdx.x;
  for (int d = threadIdx.x; d < D; d += kRowThreads)
    out[t * ldo + d] = from_float<T>(xielu_exact(to_float<T>(z[t * ldz + d]), pos, neg));
}

struct AddNormedMix {
  float* x;
  int64_t ldx;
  const void *a, *b, *rows, *same, *table;
  int64_t lda, ldb, ld_rows, ld_same, ld_table;
  float sa, sb;
  const float* gb;           // [T] per-token factor on b, or NULL
  const float* wts;          // [T, top] or NULL (1)
  const int* ids;            // [T, top] or NULL (every row is an expert's)
  int top, n_experts;
  const int64_t* table_ids;  // [T]
  const float* w;
  float eps, mult;
  void* out_h;
  int64_t ldh;
  const float* w_next;
  int W;
};

__device__ __forceinline__ float block_sum_any(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < nw ? red[l] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  return t;
}

// acc[i] += s * p[i] for the V consecutive values of one 16-byte load
template <typename TA, int V>
__device__ __forceinline__ void axpy_load(float (&acc)[V], float s, const TA* p) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const TA* e = reinterpret_cast<const TA*>(&u);
#pragma unroll
  for (int i = 0; i < V; ++i) acc[i] = fmaf(s, to_float<TA>(e[i]), acc[i]);
}

// Any width and alignment: the summed row, then the new residual row, stay in shared memory.
template <typename TA>
__global__ void __launch_bounds__(kRowThreads)
add_normed_mix_any_kernel(const AddNormedMix p) {
  extern __shared__ float mix_row[];
  __shared__ float red[kRowThreads / 32];
  const int64_t t = blockIdx.x;
  const int W = p.W;
  const float gb = p.b ? (p.gb ? p.gb[t] : 1.f) * p.sb : 0.f;
  float s = 0.f;
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    float v = 0.f;
    if (p.a) v = fmaf(p.sa, to_float<TA>(static_cast<const TA*>(p.a)[t * p.lda + d]), v);
    if (p.b) v = fmaf(gb, to_float<TA>(static_cast<const TA*>(p.b)[t * p.ldb + d]), v);
    if (p.rows)
      for (int k = 0; k < p.top; ++k) {
        const bool own = p.ids && p.ids[t * p.top + k] >= p.n_experts;
        const TA* src = own ? static_cast<const TA*>(p.same) + t * p.ld_same
                            : static_cast<const TA*>(p.rows) + (t * p.top + k) * p.ld_rows;
        v = fmaf(p.wts ? p.wts[t * p.top + k] : 1.f, to_float<TA>(src[d]), v);
      }
    mix_row[d] = v;
    s = fmaf(v, v, s);
  }
  const float r = p.mult / sqrtf(block_sum(s, red) / static_cast<float>(W) + p.eps);
  const TA* extra = p.table ? static_cast<const TA*>(p.table) + p.table_ids[t] * p.ld_table : nullptr;
  float s2 = 0.f;
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    float nx = fmaf(mix_row[d] * r, p.w ? p.w[d] : 1.f, p.x[t * p.ldx + d]);
    if (extra) nx += to_float<TA>(extra[d]);
    p.x[t * p.ldx + d] = nx;
    mix_row[d] = nx;
    s2 = fmaf(nx, nx, s2);
  }
  if (!p.out_h) return;
  const float r2 = p.w_next ? 1.0f / sqrtf(block_sum(s2, red) / static_cast<float>(W) + p.eps) : 1.f;
  for (int d = threadIdx.x; d < W; d += kRowThreads)
    static_cast<TA*>(p.out_h)[t * p.ldh + d] = from_float<TA>(mix_row[d] * r2 * (p.w_next ? p.w_next[d] : 1.f));
}

// A thread owns NC chunks of V consecutive coordinates of one token's row.
template <typename TA, int V, int NC>
__global__ void __launch_bounds__(kRowThreads)
add_normed_mix_kernel(const AddNormedMix p) {
  __shared__ float red[kRowThreads / 32];
  const int64_t t = blockIdx.x;
  const int W = p.W;
  float y[NC][V];
  float s = 0.f;
  const float gb = p.b ? (p.gb ? p.gb[t] : 1.f) * p.sb : 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int d = (c * blockDim.x + threadIdx.x) * V;
#pragma unroll
    for (int i = 0; i < V; ++i) y[c][i] = 0.f;
    if (d < W) {
      if (p.a) axpy_load<TA, V>(y[c], p.sa, static_cast<const TA*>(p.a) + t * p.lda + d);
      if (p.b) axpy_load<TA, V>(y[c], gb, static_cast<const TA*>(p.b) + t * p.ldb + d);
      if (p.rows) {
#pragma unroll 4
        for (int k = 0; k < p.top; ++k) {
          const float wk = p.wts ? p.wts[t * p.top + k] : 1.f;
          const bool own = p.ids && p.ids[t * p.top + k] >= p.n_experts;
          axpy_load<TA, V>(y[c], wk, own ? static_cast<const TA*>(p.same) + t * p.ld_same + d
                                         : static_cast<const TA*>(p.rows) + (t * p.top + k) * p.ld_rows + d);
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) s = fmaf(y[c][i], y[c][i], s);
    }
  }
  s = block_sum_any(s, red);
  const float r = p.mult / sqrtf(s / static_cast<float>(W) + p.eps);
  float s2 = 0.f;
  const TA* extra = p.table ? static_cast<const TA*>(p.table) + p.table_ids[t] * p.ld_table : nullptr;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int d = (c * blockDim.x + threadIdx.x) * V;
    if (d < W) {
      float* xr = p.x + t * p.ldx + d;
      float nx[V];
#pragma unroll
        for (int i = 0; i < V; i += 4) {
          const float4 xv = *reinterpret_cast<const float4*>(xr + i);
          const float4 wv = p.w ? *reinterpret_cast<const float4*>(p.w + d + i) : make_float4(1.f, 1.f, 1.f, 1.f);
          nx[i] = fmaf(y[c][i] * r, wv.x, xv.x);
          nx[i + 1] = fmaf(y[c][i + 1] * r, wv.y, xv.y);
          nx[i + 2] = fmaf(y[c][i + 2] * r, wv.z, xv.z);
          nx[i + 3] = fmaf(y[c][i + 3] * r, wv.w, xv.w);
        }
      if (extra) axpy_load<TA, V>(nx, 1.f, extra + d);
#pragma unroll
      for (int i = 0; i < V; i += 4)
        *reinterpret_cast<float4*>(xr + i) = make_float4(nx[i], nx[i + 1], nx[i + 2], nx[i + 3]);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        s2 = fmaf(nx[i], nx[i], s2);
        y[c][i] = nx[i];
      }
    }
  }
  if (!p.out_h) return;
  float r2 = 1.f;
  if (p.w_next) {
    s2 = block_sum_any(s2, red);
    r2 = 1.0f / sqrtf(s2 / static_cast<float>(W) + p.eps);
  }
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int d = (c * blockDim.x + threadIdx.x) * V;
    if (d >= W) continue;
    TA* dst = static_cast<TA*>(p.out_h) + t * p.ldh + d;
      uint4 u;
      TA* e = reinterpret_cast<TA*>(&u);
#pragma unroll
      for (int i = 0; i < V; i += 4) {
        const float4 wv = p.w_next ? *reinterpret_cast<const float4*>(p.w_next + d + i) : make_float4(1.f, 1.f, 1.f, 1.f);
        e[i] = from_float<TA>(y[c][i] * r2 * wv.x);
        e[i + 1] = from_float<TA>(y[c][i + 1] * r2 * wv.y);
        e[i + 2] = from_float<TA>(y[c][i + 2] * r2 * wv.z);
        e[i + 3] = from_float<TA>(y[c][i + 3] * r2 * wv.w);
      }
      *reinterpret_cast<uint4*>(dst) = u;
  }
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
softcap_rows_kernel(const T* __restrict__ z, int64_t ldz, float* __restrict__ out, int64_t ldo, int V,
                    float cap) {
  const int t = blockIdx.x;
  for (int d = threadIdx.x; d < V; d += kRowThreads) {
    const float v = to_float<T>(z[t * ldz + d]);
    out[t * ldo + d] = cap > 0.f ? cap * tanhf(v / cap) : v;
  }
}

template <typename TA, typename TO>
__global__ void __launch_bounds__(kRowThreads)
scaled_add_layernorm_kernel(float* __restrict__ x, int64_t ldx, float alpha, const TA* __restrict__ a,
                            int64_t lda, const TA* __restrict__ b, int64_t ldb,
                            const TA* __restrict__ rows, int64_t ld_rows,
                            const float* __restrict__ wts, int top, const float* __restrict__ w,
                            const float* __restrict__ bias, float eps, TO* __restrict__ out_h,
                            int64_t ldh, int W, int in_place) {
  extern __shared__ float ln_row[];          // [W] the summed row
  __shared__ float red[kRowThreads / 32];
  const int t = blockIdx.x;
  float s = 0.f;
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    float v = alpha * x[t * ldx + d];
    if (a) v += to_float<TA>(a[t * lda + d]);
    if (rows)
      for (int k = 0; k < top; ++k)
        v = fmaf(wts ? wts[t * top + k] : 1.f, to_float<TA>(rows[(static_cast<int64_t>(t) * top + k) * ld_rows + d]), v);
    if (b) v += to_float<TA>(b[t * ldb + d]);
    ln_row[d] = v;
    s += v;
  }
  const float mean = block_sum(s, red) / static_cast<float>(W);
  float q = 0.f;
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    const float c = ln_row[d] - mean;
    q = fmaf(c, c, q);
  }
  const float r = 1.0f / sqrtf(block_sum(q, red) / static_cast<float>(W) + eps);
  for (int d = threadIdx.x; d < W; d += kRowThreads) {
    const float y = fmaf((ln_row[d] - mean) * r, w ? w[d] : 1.f, bias ? bias[d] : 0.f);
    if (in_place) x[t * ldx + d] = y;
    if (out_h) out_h[t * ldh + d] = from_float<TO>(y);
  }
}

// the same, 16 bytes of gate and of up-projection per thread
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
act_and_mul_clamped_vec_kernel(const T* __restrict__ z, int64_t ldz, T* __restrict__ out, int64_t ldo, int D,
                               float limit, float slope) {
  constexpr int V = 16 / sizeof(T);
  const int64_t t = blockIdx.y;
  const int d = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (d >= D) return;
  const uint4 gu = *reinterpret_cast<const uint4*>(z + t * ldz + d);
  const uint4 uu = *reinterpret_cast<const uint4*>(z + t * ldz + D + d);
  uint4 o;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const float g = fminf(to_float<T>(reinterpret_cast<const T*>(&gu)[i]), limit);
    const float u = fminf(fmaxf(to_float<T>(reinterpret_cast<const T*>(&uu)[i]), -limit), limit);
    reinterpret_cast<T*>(&o)[i] = from_float<T>(g / (1.0f + expf(-slope * g)) * (u + 1.0f));
  }
  *reinterpret_cast<uint4*>(out + t * ldo + d) = o;
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
act_and_mul_clamped_kernel(const T* __restrict__ z, int64_t ldz, T* __restrict__ out, int64_t ldo, int D,
                           float limit, float slope) {
  const int t = blockIdx.x;
  for (int d = threadIdx.x; d < D; d += kRowThreads) {
    const float g = fminf(to_float<T>(z[t * ldz + d]), limit);
    const float u = fminf(fmaxf(to_float<T>(z[t * ldz + D + d]), -limit), limit);
    out[t * ldo + d] = from_float<T>(g / (1.0f + expf(-slope * g)) * (u + 1.0f));
  }
}

}  // namespace b200

extern "C" int b200_scalar_rmsnorm_shift(const float* x, int64_t ldx, const float* gain,
                                         const float* weight, float eps, const float* mu,
                                         float* state, int64_t ld_state, const int* tok_pos,
                                         const int* tok_b, const int* ext_start, const int* ext_len,
                                         const int64_t* slot, void* out_h, int64_t ldh, void* out_hm,
                                         int64_t ldm, int T, int W, int out_dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(x && (out_h || out_hm) && T > 0 && W > 0, "b200_scalar_rmsnorm_shift: bad arguments");
  B200_REQUIRE(!mu || (out_hm && tok_pos && tok_b && ext_start && ext_len),
               "b200_scalar_rmsnorm_shift: the shift needs out_hm and the token/portion tables");
  B200_REQUIRE(mu || out_h, "b200_scalar_rmsnorm_shift: out_h is NULL");
  B200_REQUIRE(!state || slot, "b200_scalar_rmsnorm_shift: state without slots");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("scalar_rmsnorm_shift", st);
#define LAUNCH(TO)                                                                                   \
  launch_kernel(scalar_rmsnorm_shift_kernel<TO>, dim3(T), dim3(kRowThreads), 0, st, 1, 0, x, ldx,   \
                gain, weight, eps, mu, state, ld_state, tok_pos, tok_b, ext_start, ext_len, slot,    \
                static_cast<TO*>(out_h), ldh, static_cast<TO*>(out_hm), ldm, W)
  if (out_dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (out_dtype == B200_F16) LAUNCH(__half);
  else if (out_dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_scalar_rmsnorm_shift: dtype %d", out_dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("scalar_rmsnorm_shift_kernel");
  return 0;
}

extern "C" int b200_residual_combine(float* x, int64_t ldx, const void* a, int64_t lda, const void* b,
                                     int64_t ldb, const void* y, int64_t ldy, const float* topk_w,
                                     int top, const void* s, int64_t lds, const float* gate, int T,
                                     int W, int dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(x && T > 0 && W > 0, "b200_residual_combine: bad arguments");
  B200_REQUIRE(!y || (topk_w && top > 0), "b200_residual_combine: expert rows without weights");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("residual_combine", st);
#define LAUNCH(TA)                                                                                   \
  launch_kernel(residual_combine_kernel<TA>, dim3(T), dim3(kRowThreads), 0, st, 1, 0, x, ldx,       \
                static_cast<const TA*>(a), lda, static_cast<const TA*>(b), ldb,                      \
                static_cast<const TA*>(y), ldy, topk_w, top, static_cast<const TA*>(s), lds, gate, W)
  if (dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half);
  else if (dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_residual_combine: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("residual_combine_kernel");
  return 0;
}

extern "C" int b200_act_and_mul(const void* z, int64_t ldz, void* out, int64_t ldo, int T, int D,
                                int kind, int dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(z && out && T > 0 && D > 0 && (kind == 0 || kind == 1), "b200_act_and_mul: bad arguments");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("act_and_mul", st);
#define LAUNCH(TT)                                                                                   \
  launch_kernel(act_and_mul_kernel<TT>, dim3(T), dim3(kRowThreads), 0, st, 1, 0,                    \
                static_cast<const TT*>(z), ldz, static_cast<TT*>(out), ldo, D, kind)
  if (dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half);
  else if (dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_act_and_mul: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("act_and_mul_kernel");
  return 0;
}

extern "C" int b200_add_normed_next(float* x, int64_t ldx, const void* a, int64_t lda, float sa,
                                    const void* b, int64_t ldb, float sb, const void* rows,
                                    int64_t ld_rows, int top, const float* w, float eps, float mult,
                                    void* out_h, int64_t ldh, const float* w_next, int T, int W,
                                    int dtype, void* stream) {
  return b200_add_normed_mix(x, ldx, a, lda, sa, b, ldb, sb, nullptr, rows, ld_rows, nullptr, nullptr, top, 0,
                             nullptr, 0, w, eps, mult, nullptr, 0, nullptr, out_h, ldh, w_next, T, W, dtype, stream);
}

extern "C" int b200_add_normed(float* x, int64_t ldx, const void* a, int64_t lda, float sa,
                               const void* b, int64_t ldb, float sb, const void* rows, int64_t ld_rows,
                               int top, const float* w, float eps, float mult, void* out_h, int64_t ldh,
                               int T, int W, int dtype, void* stream) {
  return b200_add_normed_next(x, ldx, a, lda, sa, b, ldb, sb, rows, ld_rows, top, w, eps, mult, out_h,
                              ldh, nullptr, T, W, dtype, stream);
}

extern "C" int b200_add_normed_mix(float* x, int64_t ldx, const void* a, int64_t lda, float sa, const void* b,
                                   int64_t ldb, float sb, const float* gb, const void* rows, int64_t ld_rows,
                                   const float* wts, const int* ids, int top, int n_experts, const void* same,
                                   int64_t ld_same, const float* w, float eps, float mult, const void* table,
                                   int64_t ld_table, const int64_t* table_ids, void* out_h, int64_t ldh,
                                   const float* w_next, int T, int W, int dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(x && (a || b || rows) && T > 0 && W > 0, "b200_add_normed_mix: bad arguments");
  B200_REQUIRE((!rows && !ids) || top > 0, "b200_add_normed_mix: rows without a count per token");
  B200_REQUIRE(!ids || (rows && same), "b200_add_normed_mix: expert ids need the expert rows and the identity rows");
  B200_REQUIRE(!w_next || out_h, "b200_add_normed_mix: a next norm without an output");
  B200_REQUIRE(!table || table_ids, "b200_add_normed_mix: a table without row ids");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("add_normed", st);
  const AddNormedMix p{x, ldx, a, b, rows, same, table, lda, ldb, ld_rows, ld_same, ld_table, sa, sb, gb, wts, ids, top,
                       n_experts, table_ids, w, eps, mult, out_h, ldh, w_next, W};
  // one 16-byte chunk per thread and pass when every row allows it
  const int v = dtype == B200_F32 ? 4 : 8;
  auto fits = [&](const void* q, int64_t ld) { return !q || (aligned16(q) && ld % v == 0); };
  const bool vec = W % v == 0 && aligned16(x) && ldx % 4 == 0 && fits(a, lda) && fits(b, ldb) && fits(rows, ld_rows) &&
                   fits(same, ld_same) && fits(table, ld_table) && fits(out_h, ldh) && aligned16(w) && aligned16(w_next) &&
                   W <= v * kRowThreads * 4;
  const int nc = W <= v * kRowThreads ? 1 : (W <= v * kRowThreads * 2 ? 2 : 4);
  const int nt = ceil_div(ceil_div(W / v, nc), 32) * 32;
  const size_t smem = sizeof(float) * static_cast<size_t>(W);
  B200_REQUIRE(vec || smem <= 200 * 1024, "b200_add_normed_mix: width %d too large", W);
#define LAUNCH(TA, V, NC) launch_kernel(add_normed_mix_kernel<TA, V, NC>, dim3(T), dim3(nt), 0, st, 1, 0, p)
#define BY_NC(TA, V)                                                                                 \
  do {                                                                                               \
    if (!vec) {                                                                                      \
      if (smem > 48 * 1024)                                                                          \
        B200_CUDA_OK(cudaFuncSetAttribute(add_normed_mix_any_kernel<TA>,                             \
                                          cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));  \
      launch_kernel(add_normed_mix_any_kernel<TA>, dim3(T), dim3(kRowThreads), smem, st, 1, 0, p);   \
    } else if (nc == 1) {                                                                            \
      LAUNCH(TA, V, 1);                                                                              \
    } else if (nc == 2) {                                                                            \
      LAUNCH(TA, V, 2);                                                                              \
    } else {                                                                                         \
      LAUNCH(TA, V, 4);                                                                              \
    }                                                                                                \
  } while (0)
  if (dtype == B200_BF16) BY_NC(__nv_bfloat16, 8);
  else if (dtype == B200_F16) BY_NC(__half, 8);
  else if (dtype == B200_F32) BY_NC(float, 4);
  else B200_REQUIRE(false, "b200_add_normed_mix: dtype %d", dtype);
#undef BY_NC
#undef LAUNCH
  B200_CHECK_LAUNCH("add_normed_mix_kernel");
  return 0;
}

extern "C" int b200_softcap_rows(const void* z, int64_t ldz, float* out, int64_t ldo, int T, int V,
                                 float cap, int dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(z && out && T > 0 && V > 0, "b200_softcap_rows: bad arguments");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("softcap_rows", st);
#define LAUNCH(TT)                                                                                   \
  launch_kernel(softcap_rows_kernel<TT>, dim3(T), dim3(kRowThreads), 0, st, 1, 0,                   \
                static_cast<const TT*>(z), ldz, out, ldo, V, cap)
  if (dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half);
  else if (dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_softcap_rows: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("softcap_rows_kernel");
  return 0;
}

extern "C" int b200_scaled_add_layernorm(float* x, int64_t ldx, float alpha, const void* a, int64_t lda,
                                         const void* b, int64_t ldb, const void* rows, int64_t ld_rows,
                                         const float* wts, int top, const float* w, const float* bias,
                                         float eps, void* out_h, int64_t ldh, int in_place, int T, int W,
                                         int dtype, int out_dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(x && T > 0 && W > 0 && (in_place || out_h), "b200_scaled_add_layernorm: bad arguments");
  B200_REQUIRE(!rows || top > 0, "b200_scaled_add_layernorm: rows without a count per token");
  B200_REQUIRE(out_dtype == dtype || out_dtype == B200_F32 || !out_h,
               "b200_scaled_add_layernorm: the copy has the terms' dtype or fp32");
  const size_t smem = sizeof(float) * static_cast<size_t>(W);
  B200_REQUIRE(smem <= 200 * 1024, "b200_scaled_add_layernorm: width %d too large", W);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("scaled_add_layernorm", st);
#define LAUNCH(TA, TO)                                                                               \
  do {                                                                                               \
    if (smem > 48 * 1024)                                                                            \
      B200_CUDA_OK(cudaFuncSetAttribute(scaled_add_layernorm_kernel<TA, TO>,                         \
                                        cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));    \
    launch_kernel(scaled_add_layernorm_kernel<TA, TO>, dim3(T), dim3(kRowThreads), smem, st, 1, 0, x, \
                  ldx, alpha, static_cast<const TA*>(a), lda, static_cast<const TA*>(b), ldb,        \
                  static_cast<const TA*>(rows), ld_rows, wts, top, w, bias, eps,                     \
                  static_cast<TO*>(out_h), ldh, W, in_place);                                        \
  } while (0)
  if (dtype == B200_BF16 && out_dtype == B200_F32) LAUNCH(__nv_bfloat16, float);
  else if (dtype == B200_F16 && out_dtype == B200_F32) LAUNCH(__half, float);
  else if (dtype == B200_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half, __half);
  else if (dtype == B200_F32) LAUNCH(float, float);
  else B200_REQUIRE(false, "b200_scaled_add_layernorm: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("scaled_add_layernorm_kernel");
  return 0;
}

extern "C" int b200_act_and_mul_clamped(const void* z, int64_t ldz, void* out, int64_t ldo, int T, int D,
                                        float limit, float slope, int dtype, void* stream) {
  using namespace b200;
  if (T == 0) return 0;
  B200_REQUIRE(z && out && T > 0 && D > 0 && limit > 0.f, "b200_act_and_mul_clamped: bad arguments");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("act_and_mul_clamped", st);
  const int v = dtype == B200_F32 ? 4 : 8;
  const bool vec = D % v == 0 && ldz % v == 0 && ldo % v == 0 && aligned16(z) && aligned16(out) && T <= 65535;
  const int nt = min(kRowThreads, ceil_div(D / v, 32) * 32);
#define LAUNCH(TT)                                                                                   \
  do {                                                                                               \
    if (vec)                                                                                         \
      launch_kernel(act_and_mul_clamped_vec_kernel<TT>, dim3(ceil_div(D / v, nt), T), dim3(nt), 0, st, 1, 0, \
                    static_cast<const TT*>(z), ldz, static_cast<TT*>(out), ldo, D, limit, slope);    \
    else                                                                                             \
      launch_kernel(act_and_mul_clamped_kernel<TT>, dim3(T), dim3(kRowThreads), 0, st, 1, 0,         \
                    static_cast<const TT*>(z), ldz, static_cast<TT*>(out), ldo, D, limit, slope);    \
  } while (0)
  if (dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half);
  else if (dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_act_and_mul_clamped: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("act_and_mul_clamped_kernel");
  return 0;
}

extern "C" int b200_xielu_rows(const void* z, int64_t ldz, void* out, int64_t ldo, int T, int D, float pos,
                               float neg, int dtype, void* stream) {
  using namespace b200;
  if (T == 0 || D == 0) return 0;
  B200_REQUIRE(z && out && T > 0 && D > 0, "b200_xielu_rows: bad arguments");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScopedKernelTimer timer("xielu_rows", st);
#define LAUNCH(TT)                                                                                   \
  launch_kernel(xielu_rows_kernel<TT>, dim3(T), dim3(kRowThreads), 0, st, 1, 0,                      \
                static_cast<const TT*>(z), ldz, static_cast<TT*>(out), ldo, D, pos, neg)
  if (dtype == B200_BF16) LAUNCH(__nv_bfloat16);
  else if (dtype == B200_F16) LAUNCH(__half);
  else if (dtype == B200_F32) LAUNCH(float);
  else B200_REQUIRE(false, "b200_xielu_rows: dtype %d", dtype);
#undef LAUNCH
  B200_CHECK_LAUNCH("xielu_rows_kernel");
  return 0;
}
