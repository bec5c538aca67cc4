// Kernels of decoders described layer by layer: what stands between the matrix products of a layer whose mixer is
// (a) attention over key/value heads with norms over the whole query / key projection, projection biases, a learned bias
// per head and distance bucket, a sliding window that keeps the first tokens, and an element-wise output gate, or
// (b) latent attention: one normed latent vector per position is cached and serves every head; a head's query is taken
// into the latent space (q' = W_uk^T q, so that q . (W_uk c) = q' . c) and its result out of it (W_uv (sum p c)).
// Heads may be rotated by their position, and a softmax may have a sink: a score without a key.
// Then the norms of the residual stream -- on a sublayer's output before its add, or on its input behind the add of the one
// before --, the gated unit, and the embedding with learned positions.  Sizes and constants are arguments; a mechanism that
// is absent is a null pointer or a zero.
//
// Scores, softmax, norms, sigmoids and the residual stream are f32 throughout.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <math_constants.h>

#include <algorithm>

#include "llr_attend.cuh"
#include "llr_kernels.cuh"

namespace llr {
namespace {

__device__ __forceinline__ float bf(uint16_t v) { return __uint_as_float((uint32_t)v << 16); }
__device__ __forceinline__ float sigmoid(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ uint2 pack4_bf16(float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  return make_uint2(*(const uint32_t*)&a, *(const uint32_t*)&b);
}

__device__ __forceinline__ float4 widen4(uint2 u) {
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}

// ---- embedding ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
embed_kernel(const uint16_t* __restrict__ table, const uint16_t* __restrict__ pos_table, const int* __restrict__ ids, RowMap rows, float scale,
             float* __restrict__ x, __nv_bfloat16* __restrict__ x16, int n, RotTable rot) {
  pdl_enter();
  const int t = blockIdx.x;
  if (rot.n > 0) {  // angles reduced in double precision: far positions keep every bit their float cosine can hold
    const double pos = (double)row_position(rows, t);
    for (int i = threadIdx.x; i < rot.n; i += blockDim.x) {
      const double turns = pos * rot.freq[i] * 0.15915494309189535;  // 1 / (2 pi)
      float sn, cs;
      sincospif((float)(2.0 * (turns - rint(turns))), &sn, &cs);
      rot.cs[(int64_t)t * rot.n + i] = make_float2(cs, sn);
    }
  }
  const uint16_t* e = table + (int64_t)ids[t] * n;
  const uint16_t* p = pos_table ? pos_table + (int64_t)row_position(rows, t) * n : nullptr;
  for (int i = 4 * threadIdx.x; i < n; i += 4 * blockDim.x) {  // n is a multiple of four
    float4 v = widen4(*(const uint2*)(e + i));
    v = make_float4(__fmul_rn(v.x, scale), __fmul_rn(v.y, scale), __fmul_rn(v.z, scale), __fmul_rn(v.w, scale));
    if (p) {
      const float4 u = widen4(*(const uint2*)(p + i));
      v = make_float4(__fadd_rn(v.x, u.x), __fadd_rn(v.y, u.y), __fadd_rn(v.z, u.z), __fadd_rn(v.w, u.w));
    }
    *(float4*)(x + (int64_t)t * n + i) = v;
    if (x16) *(uint2*)(x16 + (int64_t)t * n + i) = pack4_bf16(v);
  }
}

// ---- projections into the cache ---------------------------------------------------------------------------------
__device__ __forceinline__ int64_t slot_of(const LayerKv& kv, int seq, int pos, int64_t block, int head, int d) {
  const int b = kv.table[(int64_t)seq * kv.max_blocks + pos / kv.block_tokens];
  return (int64_t)b * block + ((int64_t)head * kv.block_tokens + pos % kv.block_tokens) * d;
}
__device__ __forceinline__ float inv_rms(float sum_sq, int n, float eps) {
  return __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(sum_sq, (float)n), eps)));
}

// A row of the stacked q | k | v projection: biases, and the factors that norm all of q and all of k.  Blocks of
// PROJ_THREADS threads; each sum is formed in one order whichever kernel asks for it.
constexpr int PROJ_THREADS = 256;
struct QkvRow {
  const float *p, *bias, *q_norm, *k_norm;
  float qi, ki;
  int nq, nk;
  __device__ __forceinline__ float q(int i) const {
    const float v = bias ? __fadd_rn(p[i], bias[i]) : p[i];
    return q_norm ? __fmul_rn(__fmul_rn(v, qi), q_norm[i]) : v;
  }
  __device__ __forceinline__ float k(int i) const {
    const float v = bias ? __fadd_rn(p[nq + i], bias[nq + i]) : p[nq + i];
    return k_norm ? __fmul_rn(__fmul_rn(v, ki), k_norm[i]) : v;
  }
  __device__ __forceinline__ float v(int i) const { return bias ? __fadd_rn(p[nq + nk + i], bias[nq + nk + i]) : p[nq + nk + i]; }
};
// a thread's share of the sum of (p + bias)^2; p and bias are 16-byte aligned and n is a multiple of four when vec
__device__ __forceinline__ float sum_squares(const float* p, const float* bias, int n, bool vec) {
  float s = 0.f;
  if (vec) {
#pragma unroll 4
    for (int i = 4 * threadIdx.x; i < n; i += 4 * PROJ_THREADS) {
      float4 v = *(const float4*)(p + i);
      if (bias) {
        const float4 u = *(const float4*)(bias + i);
        v = make_float4(__fadd_rn(v.x, u.x), __fadd_rn(v.y, u.y), __fadd_rn(v.z, u.z), __fadd_rn(v.w, u.w));
      }
      s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    }
  } else {
    for (int i = threadIdx.x; i < n; i += PROJ_THREADS) {
      const float v = bias ? __fadd_rn(p[i], bias[i]) : p[i];
      s = fmaf(v, v, s);
    }
  }
  return s;
}
__device__ __forceinline__ QkvRow qkv_row(const float* p, int ld, const float* bias, const float* q_norm, const float* k_norm, const QkvShape& sh,
                                          float (*red)[32]) {
  const int nq = sh.n_head * sh.dk, nk = sh.n_kv * sh.dk;
  const bool vec = ((ld | nq | nk) & 3) == 0;
  QkvRow r{p, bias, q_norm, k_norm, 1.f, 1.f, nq, nk};
  const float qs = q_norm ? sum_squares(p, bias, nq, vec) : 0.f, ks = k_norm ? sum_squares(p + nq, bias ? bias + nq : nullptr, nk, vec) : 0.f;
  if (q_norm) r.qi = inv_rms(block_sum(qs, red[0]), nq, sh.eps);
  if (k_norm) r.ki = inv_rms(block_sum(ks, red[1]), nk, sh.eps);
  return r;
}

// Value i of a run of heads of d values whose values before the rotation are f(i); cs: the row's cosines and sines
template <typename F>
__device__ __forceinline__ float rotated(const F& f, int i, int d, const float2* cs, int dims) {
  const int c = i % d, half = dims / 2;
  const float v = f(i);
  if (c >= dims) return v;
  const float2 a = cs[c < half ? c : c - half];
  return c < half ? fmaf(v, a.x, -__fmul_rn(f(i + half), a.y)) : fmaf(v, a.x, __fmul_rn(f(i - half), a.y));
}
// The same for `heads` whole heads, a warp per head; put(i, v) takes value i
template <typename F, typename P>
__device__ __forceinline__ void rotate_all(const F& f, const P& put, int heads, int d, const float2* cs, int dims) {
  const int half = dims / 2, lane = threadIdx.x & 31;
  for (int h = threadIdx.x >> 5; h < heads; h += blockDim.x >> 5) {
    const int i0 = h * d;
#pragma unroll 2
    for (int c = lane; c < half; c += 32) {  // a pair is read and written by one thread
      const float u = f(i0 + c), v = f(i0 + c + half);
      const float2 a = cs[c];
      put(i0 + c, fmaf(u, a.x, -__fmul_rn(v, a.y)));
      put(i0 + c + half, fmaf(v, a.x, __fmul_rn(u, a.y)));
    }
    for (int c = dims + lane; c < d; c += 32) put(i0 + c, f(i0 + c));
  }
}
__device__ __forceinline__ void rotate_heads(const RotHeads& h, int64_t ld, int t) {
  float* x = h.x + (int64_t)t * ld;
  rotate_all([&](int i) { return x[i]; }, [&](int i, float v) { x[i] = v; }, h.heads, h.dim, h.rot.cs + (int64_t)t * h.rot.ld, h.rot.dims);
}
__global__ void __launch_bounds__(256)
rotate_heads_kernel(RotHeads h, int ld) {
  pdl_enter();
  rotate_heads(h, ld, blockIdx.x);
}

// one block per row
__global__ void __launch_bounds__(PROJ_THREADS)
qkv_store_kernel(float* proj, int ld, const float* __restrict__ bias, const float* __restrict__ q_norm,
                 const float* __restrict__ k_norm, QkvShape sh, RotRows rot, RotHeads also, LayerKv kv, RowMap rows) {
  pdl_enter();
  __shared__ float red[2][32];
  const int t = blockIdx.x, nk = sh.n_kv * sh.dk, nv = sh.n_kv * sh.dv;
  float* p = proj + (int64_t)t * ld;
  const QkvRow r = qkv_row(p, ld, bias, q_norm, k_norm, sh, red);
  const int pos = row_position(rows, t), seq = row_sequence(rows, t);
  // the page and the place in it once; heads lie block_tokens vectors apart
  float* k0 = kv.k + slot_of(kv, seq, pos, kv.k_block, 0, sh.dk);
  float* v0 = kv.v + slot_of(kv, seq, pos, kv.v_block, 0, sh.dv);
  if (also.heads > 0) rotate_heads(also, ld, t);
  const float2* cs = rot.dims > 0 ? rot.cs + (int64_t)t * rot.ld : nullptr;
  const auto qf = [&](int i) { return r.q(i); };
  const auto kf = [&](int i) { return r.k(i); };
  auto k_at = [&](int i) { return k0 + (int64_t)(i / sh.dk) * kv.block_tokens * sh.dk + i % sh.dk; };
  if (cs) {
    rotate_all(kf, [&](int i, float v) { *k_at(i) = v; }, sh.n_kv, sh.dk, cs, rot.dims);
  } else {
    for (int i = threadIdx.x; i < nk; i += PROJ_THREADS) *k_at(i) = r.k(i);
  }
  for (int i = threadIdx.x; i < nv; i += PROJ_THREADS) v0[(int64_t)(i / sh.dv) * kv.block_tokens * sh.dv + i % sh.dv] = r.v(i);
  if (cs) {
    rotate_all(qf, [&](int i, float v) { p[i] = v; }, sh.n_head, sh.dk, cs, rot.dims);
  } else if (bias || q_norm) {
    for (int i0 = threadIdx.x; i0 < r.nq; i0 += 4 * PROJ_THREADS) {  // four values in flight; each is read and written by one thread
      float u[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) u[j] = i0 + j * PROJ_THREADS < r.nq ? r.q(i0 + j * PROJ_THREADS) : 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (i0 + j * PROJ_THREADS < r.nq) p[i0 + j * PROJ_THREADS] = u[j];
    }
  }
}

// the latent of a row: normed, weighted, into the cache
__device__ __forceinline__ void store_latent(const float* p, const float* w, int n, float eps, float* c, float* red) {
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += PROJ_THREADS) ss = fmaf(p[i], p[i], ss);
  const float inv = inv_rms(block_sum(ss, red), n, eps);
  for (int i = threadIdx.x; i < n; i += PROJ_THREADS) {
    const float v = __fmul_rn(p[i], inv);
    c[i] = w ? __fmul_rn(v, w[i]) : v;
  }
}
__global__ void __launch_bounds__(PROJ_THREADS)
latent_store_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ w, int n, float eps, LayerKv kv, RowMap rows) {
  pdl_enter();
  __shared__ float red[32];
  const int t = blockIdx.x;
  store_latent(proj + (int64_t)t * ld, w, n, eps, kv.k + slot_of(kv, row_sequence(rows, t), row_position(rows, t), kv.k_block, 0, n), red);
}

__global__ void __launch_bounds__(256)
rows_bf16_kernel(const float* __restrict__ x, int64_t ld, int n, __nv_bfloat16* __restrict__ o) {
  pdl_enter();
  const float* xr = x + (int64_t)blockIdx.x * ld;
  __nv_bfloat16* orow = o + (int64_t)blockIdx.x * n;
  if ((n & 3) == 0 && (ld & 3) == 0) {
    for (int i = 4 * threadIdx.x; i < n; i += 4 * blockDim.x) *(uint2*)(orow + i) = pack4_bf16(*(const float4*)(xr + i));
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) orow[i] = __float2bfloat16_rn(xr[i]);
  }
}

// ---- products per head, f32 activations ---------------------------------------------------------------------------
// y[t][h * cols + c] = sum_r W[h * rows + r][c] x[t][h * rows + r]: a thread owns two columns and every fourth row (W is
// read along its rows), the four partial sums are added in order.
template <int TT>
__global__ void __launch_bounds__(256)
head_product_t_kernel(const uint16_t* __restrict__ w, int heads, int rows, int cols, const float* __restrict__ x, int64_t x_ld,
                      float* __restrict__ y, int tokens) {
  pdl_enter();
  __shared__ float part[4][TT][128];
  const int h = blockIdx.y, t0 = blockIdx.z * TT, cp = threadIdx.x & 63, grp = threadIdx.x >> 6;
  const int c = blockIdx.x * 128 + 2 * cp;
  const bool two = c + 1 < cols, one = c < cols, pair = (cols & 1) == 0;
  float a0[TT], a1[TT];
#pragma unroll
  for (int j = 0; j < TT; ++j) a0[j] = a1[j] = 0.f;
  if (one) {
    const uint16_t* wh = w + (int64_t)h * rows * cols + c;
    const float* xh = x + (int64_t)t0 * x_ld + (int64_t)h * rows;
#pragma unroll (TT == 1 ? 16 : 8)
    for (int r = grp; r < rows; r += 4) {
      float w0, w1;
      if (pair) {
        const uint32_t u = *(const uint32_t*)(wh + (int64_t)r * cols);
        w0 = __uint_as_float(u << 16); w1 = __uint_as_float(u & 0xffff0000u);
      } else {
        w0 = bf(wh[(int64_t)r * cols]); w1 = two ? bf(wh[(int64_t)r * cols + 1]) : 0.f;
      }
#pragma unroll
      for (int j = 0; j < TT; ++j)
        if (t0 + j < tokens) {
          const float xv = xh[(int64_t)j * x_ld + r];
          a0[j] = fmaf(w0, xv, a0[j]);
          a1[j] = fmaf(w1, xv, a1[j]);
        }
    }
  }
#pragma unroll
  for (int j = 0; j < TT; ++j) { part[grp][j][2 * cp] = a0[j]; part[grp][j][2 * cp + 1] = a1[j]; }
  __syncthreads();
  for (int i = threadIdx.x; i < TT * 128; i += 256) {
    const int j = i >> 7, k = i & 127, col = blockIdx.x * 128 + k;
    if (t0 + j < tokens && col < cols)
      y[(int64_t)(t0 + j) * heads * cols + (int64_t)h * cols + col] = (part[0][j][k] + part[1][j][k]) + (part[2][j][k] + part[3][j][k]);
  }
}

// y[t][h * rows + r] = sum_c W[h * rows + r][c] x[t][h * cols + c], times the head's gate: one warp per row of W
template <int TT>
__global__ void __launch_bounds__(256)
head_product_kernel(const uint16_t* __restrict__ w, int heads, int rows, int cols, const float* __restrict__ x, int64_t x_ld,
                    float* __restrict__ y, const float* __restrict__ gate, int64_t gate_ld, int tokens) {
  pdl_enter();
  const int lane = threadIdx.x & 31, row = blockIdx.x * 8 + (threadIdx.x >> 5), t0 = blockIdx.y * TT;
  if (row >= heads * rows) return;
  const int h = row / rows;
  const uint16_t* wr = w + (int64_t)row * cols;
  const float* xh = x + (int64_t)t0 * x_ld + (int64_t)h * cols;
  float acc[TT];
#pragma unroll
  for (int j = 0; j < TT; ++j) acc[j] = 0.f;
  if ((cols & 3) == 0 && (x_ld & 3) == 0 && ((uintptr_t)x & 15) == 0) {
#pragma unroll 4
    for (int c = 4 * lane; c < cols; c += 128) {
      const uint2 u = *(const uint2*)(wr + c);
      const float w0 = __uint_as_float(u.x << 16), w1 = __uint_as_float(u.x & 0xffff0000u), w2 = __uint_as_float(u.y << 16),
                  w3 = __uint_as_float(u.y & 0xffff0000u);
#pragma unroll
      for (int j = 0; j < TT; ++j)
        if (t0 + j < tokens) {
          const float4 v = *(const float4*)(xh + (int64_t)j * x_ld + c);
          acc[j] = fmaf(w0, v.x, fmaf(w1, v.y, fmaf(w2, v.z, fmaf(w3, v.w, acc[j]))));
        }
    }
  } else {
    for (int c = lane; c < cols; c += 32) {
      const float wv = bf(wr[c]);
#pragma unroll
      for (int j = 0; j < TT; ++j)
        if (t0 + j < tokens) acc[j] = fmaf(wv, xh[(int64_t)j * x_ld + c], acc[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < TT; ++j) {
    const float v = warp_sum(acc[j]);
    if (lane == 0 && t0 + j < tokens) {
      const int64_t t = t0 + j;
      y[t * heads * rows + row] = gate ? __fmul_rn(v, sigmoid(gate[t * gate_ld + h])) : v;
    }
  }
}

// out[h * cols + c][r] = w[h * rows + r][c] (once per session)
__global__ void head_transpose_kernel(const uint16_t* __restrict__ w, int rows, int cols, uint16_t* __restrict__ out) {
  const int64_t n = (int64_t)rows * cols, base = (int64_t)blockIdx.y * n;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x)
    out[base + (i % cols) * rows + i / cols] = w[base + i];
}

// ---- attention --------------------------------------------------------------------------------------------------
// The keys position pos sees, as one ascending list: the kept first tokens that lie before the window, then the window.
struct Span {
  int lo, nk, n;  // first position of the window, kept tokens before it, visible keys
  __device__ __forceinline__ int at(int m) const { return m < nk ? m : lo + m - nk; }
};
__device__ __forceinline__ Span span_of(int pos, int window, int keep_first) {
  const int lo = window > 0 ? max(0, pos - window + 1) : 0, nk = min(keep_first, lo);
  return Span{lo, nk, nk + pos - lo + 1};
}

struct KvSpan {
  const LayerKv& kv;
  const SpanShape& sh;
  const int2* where;  // page and place in it of the slice's keys, looked up once
  Span span;
  int s0, head, pos, h0;  // first key of the slice, kv head, the row's position, first query head
  __device__ __forceinline__ const float* k(int m) const {
    const int2 w = where[m - s0];
    return kv.k + w.x * kv.k_block + (int64_t)(head * kv.block_tokens + w.y) * sh.dk;
  }
  __device__ __forceinline__ const float* v(int m) const {
    const int2 w = where[m - s0];
    return kv.v + w.x * kv.v_block + (int64_t)(head * kv.block_tokens + w.y) * sh.dv;
  }
  __device__ __forceinline__ float score(int g, int m, float dot) const {
    const float s = __fmul_rn(dot, sh.scale);
    return sh.bias ? __fadd_rn(s, sh.bias[(int64_t)(h0 + g) * sh.bias_len + min(pos - span.at(m), sh.bias_len - 1)]) : s;
  }
};

// Keys of a slice for a row that sees n of them: 32 slices once there are enough keys, so that a short sequence in a long
// context still spreads over the SMs.  Never more than the chunk the launch is sized for.
__device__ __forceinline__ int span_step(int n) { return max(32, (n + 31) / 32); }

// Query heads of a kv head that share a block: eight, four where a head's query and value rows are long.
inline __host__ __device__ int span_heads(const SpanShape& sh) { return sh.dk + sh.dv > 512 ? ATT_MAX_GQA / 2 : ATT_MAX_GQA; }

// grid (kv head x group of span_heads query heads, slice of the visible keys, row)
// With nt (a single decode token) the kernel also does what the store kernels do for that token: the query is biased and
// normed as it is loaded, and the blocks whose slice holds the token's own position write its key and value (or its
// latent) into the cache and read them back like any other; blocks that share a kv head write the same values.
static_assert(PROJ_THREADS == ATT_THREADS, "the sums over a projection are formed in one order");
template <int MAX_VALUE>
__global__ void __launch_bounds__(ATT_THREADS)
span_partial_kernel(const float* __restrict__ q, int64_t q_ld, SpanShape sh, LayerKv kv, RowMap rows, int t0, int chunk, float* __restrict__ part,
                    NewToken nt) {
  pdl_enter();
  __shared__ float red[2][32];
  extern __shared__ int2 smw[];  // pages [chunk] | q [heads][dk] | scores [heads][chunk] or sums [P][heads][dv]
  float* sm = (float*)(smw + chunk);
  const int gq = sh.n_head / sh.n_kv, per = span_heads(sh), groups = (gq + per - 1) / per;
  const int head = blockIdx.x / groups, g0 = (blockIdx.x % groups) * per, heads = min(per, gq - g0);
  const int t = t0 + blockIdx.z, split = blockIdx.y, n_split = (int)gridDim.y, h0 = head * gq + g0;
  const int pos = row_position(rows, t);
  const Span span = span_of(pos, sh.window, sh.keep_first);
  const int step = span_step(span.n), s0 = split * step, s1 = min(span.n, s0 + step);
  if (s0 >= span.n) return;
  float* sq = sm;
  float* sc = sq + heads * sh.dk;
  for (int m = s0 + threadIdx.x; m < s1; m += ATT_THREADS) {
    const int j = span.at(m);
    smw[m - s0] = make_int2(kv.table[(int64_t)row_sequence(rows, t) * kv.max_blocks + j / kv.block_tokens], j % kv.block_tokens);
  }
  if (nt.proj && !nt.latent) {
    const QkvShape qs{sh.n_head, sh.n_kv, sh.dk, sh.dv, nt.eps};
    const QkvRow r = qkv_row(nt.proj, (int)q_ld, nt.bias, nt.q_norm, nt.k_norm, qs, red);
    const float2* cs = nt.rot.dims > 0 ? nt.rot.cs + (int64_t)t * nt.rot.ld : nullptr;
    const auto qf = [&](int i) { return r.q(i); };
    const auto kf = [&](int i) { return r.k(i); };
    for (int i = threadIdx.x; i < heads * sh.dk; i += ATT_THREADS)
      sq[i] = cs ? rotated(qf, h0 * sh.dk + i, sh.dk, cs, nt.rot.dims) : r.q(h0 * sh.dk + i);
    if (s1 == span.n) {
      float* k = kv.k + slot_of(kv, row_sequence(rows, t), pos, kv.k_block, head, sh.dk);
      float* v = kv.v + slot_of(kv, row_sequence(rows, t), pos, kv.v_block, head, sh.dv);
      for (int i = threadIdx.x; i < sh.dk; i += ATT_THREADS)
        k[i] = cs ? rotated(kf, head * sh.dk + i, sh.dk, cs, nt.rot.dims) : r.k(head * sh.dk + i);
      for (int i = threadIdx.x; i < sh.dv; i += ATT_THREADS) v[i] = r.v(head * sh.dv + i);
    }
  } else {
    for (int i = threadIdx.x; i < heads * sh.dk; i += ATT_THREADS) sq[i] = q[(int64_t)t * q_ld + (int64_t)h0 * sh.dk + i];
    if (nt.proj && s1 == span.n) store_latent(nt.proj, nt.k_norm, sh.dk, nt.eps, kv.k + slot_of(kv, row_sequence(rows, t), pos, kv.k_block, 0, sh.dk), red[0]);
  }
  __syncthreads();
  // records: [row of the pass][query head][slice][dv + 2]; a group's heads follow each other n_split records apart
  float* rec = part + (((int64_t)blockIdx.z * sh.n_kv * groups + blockIdx.x) * n_split + split) * per * (sh.dv + 2);
  attend_slice<MAX_VALUE>(KvSpan{kv, sh, smw, span, s0, head, pos, h0}, sq, sc, rec, s0, s1, chunk, sh.dk, sh.dv, heads);
}

// grid (query head, row, 128 dimensions): merges a head's slices (at most 32) and the sink, applies the gate
__global__ void __launch_bounds__(128)
span_combine_kernel(const float* __restrict__ part, SpanShape sh, RowMap rows, int t0, int n_split, SpanOut so) {
  pdl_enter();
  const int lane = threadIdx.x & 31, h = blockIdx.x, t = t0 + blockIdx.y;
  const int gq = sh.n_head / sh.n_kv, per = span_heads(sh), groups = (gq + per - 1) / per;
  const int bx = (h / gq) * groups + (h % gq) / per, g = (h % gq) % per;
  const int seen = span_of(row_position(rows, t), sh.window, sh.keep_first).n, step = span_step(seen), used = (seen + step - 1) / step;
  const int64_t stride = (int64_t)per * (sh.dv + 2);
  const float* base = part + ((int64_t)blockIdx.y * sh.n_kv * groups + bx) * n_split * stride + g * (sh.dv + 2);
  const float ms = lane < used ? base[lane * stride + sh.dv] : -CUDART_INF_F;
  float m = warp_max(ms);
  if (sh.sink) m = fmaxf(m, sh.sink[h]);
  const float e = lane < used ? expf(ms - m) : 0.f;
  float l = warp_sum(lane < used ? base[lane * stride + sh.dv + 1] * e : 0.f);
  if (sh.sink) l = __fadd_rn(l, expf(sh.sink[h] - m));
  const int i = blockIdx.z * 128 + threadIdx.x;
  const bool live = i < sh.dv;
  float acc = 0.f;
  for (int sp = 0; sp < used; sp += 8) {  // eight slices' values are fetched before the first is used
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = (live && sp + j < used) ? base[(sp + j) * stride + i] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) acc = fmaf(v[j], __shfl_sync(~0u, e, (sp + j) & 31), acc);  // a slice beyond `used` has value 0 and weight 0
  }
  if (live) {
    float r = __fdiv_rn(acc, l);
    const int64_t o = (int64_t)h * sh.dv + i;
    if (so.gate) r = __fmul_rn(r, sigmoid(so.gate[(int64_t)t * so.gate_ld + (so.head_gate ? h : o)]));
    r = __fmul_rn(r, so.scale);
    if (so.out) so.out[(int64_t)t * so.ld + o] = r;
    if (so.out16) ((__nv_bfloat16*)so.out16)[(int64_t)t * so.ld + o] = __float2bfloat16_rn(r);
  }
}

// ---- prompt chunks on the tensor cores ------------------------------------------------------------------------------
// Rows of ONE sequence at consecutive positions.  The keys and values that any of the rows sees are first gathered from
// their pages into contiguous binary16 rows (span_gather_kernel), so that the attention kernel copies tiles with 16-byte
// asynchronous copies and neither looks pages up nor converts.
// A block takes one kv head and 64 (row, query head) pairs in row-major order -- all query heads of a kv head share its
// keys, so any ratio of heads fills the tile (one latent for every head included) -- and walks the keys that any of its
// rows sees, 64 at a time.  Queries (rescaled per pair by a power of two), keys, values and the exponentials are
// binary16 operands; scores and sums are m16n8k16 MMAs with f32 accumulators; scale, distance bias, mask, maxima,
// exponentials and their sums are f32.
// Sixteen pairs belong to NS warps: each scores 64 / NS of the keys and owns 8 ND of the value dimensions.
// The copies run one tile ahead of their use: values arrive while their keys are scored, the next keys while the values
// are added up; where keys and values are one latent there are two buffers instead.
constexpr int CH = 64;
__device__ __forceinline__ uint32_t pack_h2(float lo, float hi) {
  const __half2 h = __floats2half2_rn(lo, hi);
  return *(const uint32_t*)&h;
}
__device__ __forceinline__ float sat16(float v) { return fminf(fmaxf(v, -65504.f), 65504.f); }
__device__ __forceinline__ void mma_f16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const __half* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void ldm4_t(uint32_t (&r)[4], const __half* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void copy16(const __half* dst, const __half* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Widths of the gathered rows and of the tiles, in halves; multiples of 16, so that a tile's pitch (width + 8) is an odd
// number of 16-byte units.  Where values are the keys there is one row of the wider of the two.
struct MmaLayout {
  int kw, vw, kr, vr;  // score columns, value columns, gathered key row, gathered value row (0: the keys)
  bool shared;
  int qp, kp, vp;
};
inline __host__ __device__ MmaLayout mma_layout(int dk, int dv, int nd, int ns, bool shared) {
  MmaLayout L;
  L.kw = (dk + 15) / 16 * 16;
  L.vw = 8 * nd * ns;
  L.shared = shared;
  L.kr = shared && L.vw > L.kw ? L.vw : L.kw;
  L.vr = shared ? 0 : L.vw;
  L.qp = L.kw + 8;
  L.kp = L.kr + 8;
  L.vp = shared ? L.kp : L.vw + 8;
  return L;
}
inline __host__ __device__ size_t mma_smem(const MmaLayout& L, int ns) {
  return ((size_t)64 * L.qp + (size_t)CH * L.kp * (L.shared ? 2 : 1) + (L.shared ? 0 : (size_t)CH * L.vp) + (ns > 1 ? 64 * (CH + 8) : 0)) * 2;
}

// The list of keys a group of rows sees: kept tokens before the first row's window, then every position from there to the
// last row.  Row m of the gathered keys of kv head g starts at k16 + ((int64_t)g * n + m) * kr.
struct GroupKeys {
  int lo, nk, n;
  __device__ __forceinline__ int at(int m) const { return m < nk ? m : lo + m - nk; }
  __device__ __forceinline__ int index(int j) const { return j < nk ? j : j - lo + nk; }  // of a position in the list
};
__device__ __forceinline__ GroupKeys group_keys(int first, int rows, int window, int keep_first) {
  const int lo = window > 0 ? max(0, first - window + 1) : 0, nk = min(keep_first, lo);
  return GroupKeys{lo, nk, nk + first + rows - lo};
}

// one warp per key row: grid (keys / 8, kv head)
__global__ void __launch_bounds__(256)
span_gather_kernel(SpanShape sh, LayerKv kv, RowMap rows, int t0, int tokens, int kr, int vr, __half* __restrict__ k16, __half* __restrict__ v16) {
  pdl_enter();
  const GroupKeys gk = group_keys(row_position(rows, t0), tokens, sh.window, sh.keep_first);
  const int m = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, head = blockIdx.y, seq = row_sequence(rows, t0);
  if (m >= gk.n) return;
  auto put = [&](const float* src, int d, __half* dst, int w) {
    for (int i = 4 * lane; i < w; i += 128) {
      const float4 v = i < d ? *(const float4*)(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);  // d is a multiple of four
      *(uint2*)(dst + i) = make_uint2(pack_h2(sat16(v.x), sat16(v.y)), pack_h2(sat16(v.z), sat16(v.w)));
    }
  };
  const int j = gk.at(m);
  put(kv.k + slot_of(kv, seq, j, kv.k_block, head, sh.dk), sh.dk, k16 + ((int64_t)head * gk.n + m) * kr, kr);
  if (vr) put(kv.v + slot_of(kv, seq, j, kv.v_block, head, sh.dv), sh.dv, v16 + ((int64_t)head * gk.n + m) * vr, vr);
}

template <int ND, int NS>
__global__ void __launch_bounds__(128 * NS)
span_mma_kernel(const float* __restrict__ q, int64_t q_ld, SpanShape sh, const __half* __restrict__ k16, const __half* __restrict__ v16, bool shared_kv,
                RowMap rows, int t0, int tokens, SpanOut so) {
  pdl_enter();
  constexpr int THR = 128 * NS, NT = CH / 8 / NS;  // score tiles of eight keys per warp
  static_assert(NT % 2 == 0, "keys are loaded sixteen at a time");
  extern __shared__ __align__(16) unsigned char raw[];
  const MmaLayout L = mma_layout(sh.dk, sh.dv, ND, NS, shared_kv);
  __half* sq = (__half*)raw;
  __half* sk = sq + 64 * L.qp;                                         // keys (two buffers where they are the values)
  __half* sv = sk + CH * L.kp;                                         // values, or the second buffer
  __half* sp = sv + CH * L.vp;                                         // exponentials, NS > 1
  __shared__ float s_scale[64], s_red[NS][64];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int rw = warp & 3, ns = warp >> 2;  // rows 16 rw .., key and value share ns
  // the last rows first: in a window that is still filling they see the most keys
  const int head = blockIdx.y, gq = sh.n_head / sh.n_kv, pairs = tokens * gq, pair0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * 64;
  const int p_first = row_position(rows, t0);
  const GroupKeys gk = group_keys(p_first, tokens, sh.window, sh.keep_first);
  const int pa = p_first + pair0 / gq, pb = p_first + min(pairs - 1, pair0 + 63) / gq;  // positions of the tile's rows
  const int lo = sh.window > 0 ? max(0, pa - sh.window + 1) : 0, nk = min(sh.keep_first, lo), n_keys = nk + pb - lo + 1;
  k16 += (int64_t)head * gk.n * L.kr;
  v16 += (int64_t)head * gk.n * L.vr;

  // rows c * CH .. of the tile's own list; rows behind its end repeat the last one (their exponentials are zero)
  auto stage = [&](__half* dst, const __half* src, int width, int pitch, int c) {
    for (int p = tid >> 4; p < CH; p += THR / 16) {
      const int m = min(c * CH + p, n_keys - 1);
      const __half* row = src + (int64_t)gk.index(m < nk ? m : lo + m - nk) * width;
      for (int d = 8 * (tid & 15); d < width; d += 128) copy16(dst + p * pitch + d, row + d);
    }
  };
  stage(sk, k16, L.kr, L.kp, 0);
  copy_commit();
  // queries: a warp per pair; the power of two that brings the largest magnitude into [2^9, 2^10)
  for (int r = warp; r < 64; r += 4 * NS) {
    const int p = pair0 + r;
    const bool live = p < pairs;
    const float* src = q + (int64_t)(t0 + (live ? p / gq : 0)) * q_ld + (int64_t)(head * gq + (live ? p % gq : 0)) * sh.dk;
    float m = 0.f;
    if (live) for (int i = lane; i < sh.dk; i += 32) m = fmaxf(m, fabsf(src[i]));
    m = warp_max(m);
    const int be = (int)((__float_as_uint(m) >> 23) & 0xff);
    const int e = (be == 0 || be == 255) ? 0 : min(126, max(-126, 136 - be));
    const float up = __uint_as_float((uint32_t)(127 + e) << 23), down = __uint_as_float((uint32_t)(127 - e) << 23);
    for (int i = lane; i < L.kw; i += 32) sq[r * L.qp + i] = __float2half_rn(live && i < sh.dk ? sat16(src[i] * up) : 0.f);
    if (lane == 0) s_scale[r] = down * sh.scale;
  }
  __syncthreads();

  constexpr float LOG2E = 1.4426950408889634f;  // scores are kept in units of ln 2: exp(x) = exp2(x log2 e)
  const int r0 = 16 * rw + g, r1 = r0 + 8;
  const int i0 = p_first + min(pair0 + r0, pairs - 1) / gq, i1 = p_first + min(pair0 + r1, pairs - 1) / gq;  // positions of this thread's rows
  const int i_lo = p_first + min(pair0 + 16 * rw, pairs - 1) / gq, i_hi = p_first + min(pair0 + 16 * rw + 15, pairs - 1) / gq;  // of this warp's
  const float* b0 = sh.bias ? sh.bias + (int64_t)(head * gq + min(pair0 + r0, pairs - 1) % gq) * sh.bias_len : nullptr;
  const float* b1 = sh.bias ? sh.bias + (int64_t)(head * gq + min(pair0 + r1, pairs - 1) % gq) * sh.bias_len : nullptr;
  const float far0 = b0 ? b0[sh.bias_len - 1] * LOG2E : 0.f, far1 = b1 ? b1[sh.bias_len - 1] * LOG2E : 0.f;
  const float f0 = s_scale[r0] * LOG2E, f1 = s_scale[r1] * LOG2E;
  float m0 = -CUDART_INF_F, m1 = -CUDART_INF_F, l0 = 0.f, l1 = 0.f;
  if (sh.sink) {  // the sink is the first score: the maximum starts there, and one thread of a row's counts it
    m0 = sh.sink[head * gq + min(pair0 + r0, pairs - 1) % gq] * LOG2E;
    m1 = sh.sink[head * gq + min(pair0 + r1, pairs - 1) % gq] * LOG2E;
    l0 = l1 = t4 == 0 && ns == 0 ? 1.f : 0.f;
  }
  float o[ND][4];
#pragma unroll
  for (int nd = 0; nd < ND; ++nd)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[nd][i] = 0.f;

  auto row_group = [&] {  // the NS warps of sixteen pairs
    if constexpr (NS == 1) __syncwarp();
    else asm volatile("bar.sync %0, %1;" ::"r"(1 + rw), "r"(32 * NS) : "memory");
  };
  const int chunks = (n_keys + CH - 1) / CH;
  for (int c = 0; c < chunks; ++c) {
    __half* kt = L.shared && (c & 1) ? sv : sk;
    __half* vt = L.shared ? kt : sv;
    if (L.shared) {
      if (c + 1 < chunks) { stage((c & 1) ? sk : sv, k16, L.kr, L.kp, c + 1); copy_commit(); copy_wait<1>(); }
      else copy_wait<0>();
    } else {
      stage(sv, v16, L.vr, L.vp, c);
      copy_commit();
      copy_wait<1>();  // the keys
    }
    __syncthreads();
    // ---- scores of this warp's keys
    float s[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int i = 0; i < 4; ++i) s[nt][i] = 0.f;
    const __half* qa = sq + (16 * rw + (lane & 15)) * L.qp + (lane >> 4) * 8;
    const __half* kb = kt + (ns * 8 * NT + (lane & 7) + (lane >> 4) * 8) * L.kp + ((lane >> 3) & 1) * 8;
#pragma unroll 2
    for (int k0 = 0; k0 < L.kw; k0 += 16) {
      uint32_t a[4];
      ldm4(a, qa + k0);
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t b[4];
        ldm4(b, kb + nt * 8 * L.kp + k0);
        mma_f16(s[nt], a, b[0], b[1]);
        mma_f16(s[nt + 1], a, b[2], b[3]);
      }
    }
    // this warp's keys of the chunk: positions between j_lo and j_hi (ascending list)
    const int k_lo = c * CH + ns * 8 * NT, k_hi = k_lo + 8 * NT - 1;
    const int j_lo = k_lo < nk ? k_lo : lo + k_lo - nk, j_hi = k_hi < nk ? k_hi : lo + k_hi - nk;
    const bool all_seen = k_hi < n_keys && j_hi <= i_lo && (sh.window <= 0 || i_hi - j_lo < sh.window || j_hi < sh.keep_first);
    const bool all_far = i_lo - j_hi >= sh.bias_len - 1;
    float x0 = -CUDART_INF_F, x1 = -CUDART_INF_F;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int m = k_lo + 8 * nt + 2 * t4 + i, j = m < nk ? m : lo + m - nk;
        float u0 = fmaf(s[nt][i], f0, far0), u1 = fmaf(s[nt][2 + i], f1, far1);
        if (!all_far || !all_seen) {  // warp-uniform
          const int d0 = i0 - j, d1 = i1 - j;
          if (b0 && !all_far) {
            u0 = fmaf(s[nt][i], f0, __ldg(b0 + min(max(d0, 0), sh.bias_len - 1)) * LOG2E);
            u1 = fmaf(s[nt][2 + i], f1, __ldg(b1 + min(max(d1, 0), sh.bias_len - 1)) * LOG2E);
          }
          const bool any = m < n_keys, kept = j < sh.keep_first || sh.window <= 0;
          if (!(any && d0 >= 0 && (kept || d0 < sh.window))) u0 = -CUDART_INF_F;
          if (!(any && d1 >= 0 && (kept || d1 < sh.window))) u1 = -CUDART_INF_F;
        }
        s[nt][i] = u0;
        s[nt][2 + i] = u1;
        x0 = fmaxf(x0, u0);
        x1 = fmaxf(x1, u1);
      }
    x0 = fmaxf(x0, __shfl_xor_sync(~0u, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(~0u, x0, 2));
    x1 = fmaxf(x1, __shfl_xor_sync(~0u, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(~0u, x1, 2));
    if constexpr (NS > 1) {
      if (t4 == 0) { s_red[ns][r0] = x0; s_red[ns][r1] = x1; }
      row_group();
#pragma unroll
      for (int k = 0; k < NS; ++k) { x0 = fmaxf(x0, s_red[k][r0]); x1 = fmaxf(x1, s_red[k][r1]); }
    }
    x0 = fmaxf(x0, m0);
    x1 = fmaxf(x1, m1);
    const float w0 = m0 == -CUDART_INF_F ? 0.f : exp2f(m0 - x0), w1 = m1 == -CUDART_INF_F ? 0.f : exp2f(m1 - x1);
    m0 = x0;
    m1 = x1;
    // a row that has seen nothing yet: every score is -inf and so is the maximum; its exponentials are zero
    const float c0 = m0 == -CUDART_INF_F ? 0.f : m0, c1 = m1 == -CUDART_INF_F ? 0.f : m1;
    l0 *= w0;
    l1 *= w1;
#pragma unroll
    for (int nd = 0; nd < ND; ++nd) { o[nd][0] *= w0; o[nd][1] *= w0; o[nd][2] *= w1; o[nd][3] *= w1; }
    uint32_t e0[NT], e1[NT];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      e0[nt] = pack_h2(exp2f(s[nt][0] - c0), exp2f(s[nt][1] - c0));
      e1[nt] = pack_h2(exp2f(s[nt][2] - c1), exp2f(s[nt][3] - c1));
      const __half2 h0 = *(const __half2*)&e0[nt], h1 = *(const __half2*)&e1[nt];
      l0 += __low2float(h0) + __high2float(h0);  // the sum of what the weighted sum below uses
      l1 += __low2float(h1) + __high2float(h1);
      if constexpr (NS > 1) {
        *(uint32_t*)(sp + r0 * (CH + 8) + ns * 8 * NT + 8 * nt + 2 * t4) = e0[nt];
        *(uint32_t*)(sp + r1 * (CH + 8) + ns * 8 * NT + 8 * nt + 2 * t4) = e1[nt];
      }
    }
    if constexpr (NS > 1) row_group();
    if (!L.shared) {
      copy_wait<0>();   // the values
      __syncthreads();  // everyone's, and every warp is done with the keys
      if (c + 1 < chunks) { stage(sk, k16, L.kr, L.kp, c + 1); copy_commit(); }
    }
    // ---- weighted values: this warp's dimensions over all keys of the chunk
    const __half* vb = vt + (lane & 15) * L.vp + ns * 8 * ND + (lane >> 4) * 8;
#pragma unroll
    for (int k0 = 0; k0 < CH; k0 += 16) {
      uint32_t a[4];
      if constexpr (NS == 1) {
        a[0] = e0[k0 / 8]; a[1] = e1[k0 / 8]; a[2] = e0[k0 / 8 + 1]; a[3] = e1[k0 / 8 + 1];
      } else {
        ldm4(a, sp + (16 * rw + (lane & 15)) * (CH + 8) + k0 + (lane >> 4) * 8);
      }
#pragma unroll
      for (int nd = 0; nd < ND; nd += 2) {
        uint32_t b[4];
        ldm4_t(b, vb + k0 * L.vp + 8 * nd);
        mma_f16(o[nd], a, b[0], b[1]);
        mma_f16(o[nd + 1], a, b[2], b[3]);
      }
    }
    __syncthreads();  // the next copies overwrite the values
  }
  l0 += __shfl_xor_sync(~0u, l0, 1); l0 += __shfl_xor_sync(~0u, l0, 2);
  l1 += __shfl_xor_sync(~0u, l1, 1); l1 += __shfl_xor_sync(~0u, l1, 2);
  if constexpr (NS > 1) {
    if (t4 == 0) { s_red[ns][r0] = l0; s_red[ns][r1] = l1; }
    row_group();
    l0 = l1 = 0.f;
#pragma unroll
    for (int k = 0; k < NS; ++k) { l0 += s_red[k][r0]; l1 += s_red[k][r1]; }
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int p = pair0 + (half ? r1 : r0);
    if (p >= pairs) continue;
    const int t = t0 + p / gq, h = head * gq + p % gq;
    float inv = __fdiv_rn(1.0f, half ? l1 : l0) * so.scale;
    if (so.gate && so.head_gate) inv *= sigmoid(so.gate[(int64_t)t * so.gate_ld + h]);
    const int64_t base = (int64_t)h * sh.dv;
#pragma unroll
    for (int nd = 0; nd < ND; ++nd) {
      const int d = ns * 8 * ND + 8 * nd + 2 * t4;
      if (d >= sh.dv) continue;
      float2 v = make_float2(o[nd][2 * half] * inv, o[nd][2 * half + 1] * inv);
      if (so.gate && !so.head_gate) {
        const float2 gg = *(const float2*)(so.gate + (int64_t)t * so.gate_ld + base + d);
        v.x *= sigmoid(gg.x);
        v.y *= sigmoid(gg.y);
      }
      const int64_t at = (int64_t)t * so.ld + base + d;
      if (so.out) *(float2*)(so.out + at) = v;
      if (so.out16) *(__nv_bfloat162*)((__nv_bfloat16*)so.out16 + at) = __floats2bfloat162_rn(v.x, v.y);
    }
  }
}

// ---- norm on a sublayer's output, residual add ------------------------------------------------------------------------
constexpr int NORM_ADD_THREADS = 512, NORM_ADD_KEEP = 4;  // up to 8192 values of a row stay in registers
__global__ void __launch_bounds__(NORM_ADD_THREADS)
norm_add_kernel(float* __restrict__ x, const float* __restrict__ y, int slices, int64_t slice_stride, const float* __restrict__ w, float eps,
                __nv_bfloat16* __restrict__ x16, int n) {
  pdl_enter();
  __shared__ float sh[32];
  float* xr = x + (int64_t)blockIdx.x * n;
  const float* yr = y + (int64_t)blockIdx.x * n;
  __nv_bfloat16* x16r = x16 ? x16 + (int64_t)blockIdx.x * n : nullptr;
  if (n % 4 == 0 && n <= 4 * NORM_ADD_THREADS * NORM_ADD_KEEP) {
    float4 keep[NORM_ADD_KEEP];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NORM_ADD_KEEP; ++k) {
      const int i = 4 * (threadIdx.x + k * NORM_ADD_THREADS);
      if (i < n) {
        float4 v = *(const float4*)(yr + i);
        for (int s = 1; s < slices; ++s) {
          const float4 u = *(const float4*)(yr + s * slice_stride + i);
          v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
        }
        keep[k] = v;
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
      }
    }
    const float inv = inv_rms(block_sum(ss, sh), n, eps);
#pragma unroll
    for (int k = 0; k < NORM_ADD_KEEP; ++k) {
      const int i = 4 * (threadIdx.x + k * NORM_ADD_THREADS);
      if (i < n) {
        const float4 ww = *(const float4*)(w + i);
        float4 r = *(const float4*)(xr + i);
        r.x = __fadd_rn(r.x, __fmul_rn(__fmul_rn(keep[k].x, inv), ww.x));
        r.y = __fadd_rn(r.y, __fmul_rn(__fmul_rn(keep[k].y, inv), ww.y));
        r.z = __fadd_rn(r.z, __fmul_rn(__fmul_rn(keep[k].z, inv), ww.z));
        r.w = __fadd_rn(r.w, __fmul_rn(__fmul_rn(keep[k].w, inv), ww.w));
        *(float4*)(xr + i) = r;
        if (x16r) *(uint2*)(x16r + i) = pack4_bf16(r);
      }
    }
    return;
  }
  auto value = [&](int i) {
    float v = yr[i];
    for (int s = 1; s < slices; ++s) v += yr[s * slice_stride + i];
    return v;
  };
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = value(i); ss = fmaf(v, v, ss); }
  const float inv = inv_rms(block_sum(ss, sh), n, eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float r = __fadd_rn(xr[i], __fmul_rn(__fmul_rn(value(i), inv), w[i]));
    xr[i] = r;
    if (x16r) x16r[i] = __float2bfloat16_rn(r);
  }
}

// ---- residual add, norm of the sum: what a sublayer reads ------------------------------------------------------------
__global__ void __launch_bounds__(NORM_ADD_THREADS)
add_norm_kernel(float* __restrict__ x, const float* __restrict__ y, int slices, int64_t slice_stride, const float* __restrict__ w, float eps,
                float* __restrict__ h, __nv_bfloat16* __restrict__ h16, int n) {
  pdl_enter();
  __shared__ float sh[32];
  const int64_t row = (int64_t)blockIdx.x * n;
  const bool in_regs = n <= 4 * NORM_ADD_THREADS * NORM_ADD_KEEP;  // n is a multiple of four
  auto fresh = [&](int i) {  // the new residual values
    float4 v = *(const float4*)(x + row + i);
    if (slices > 0) {
      float4 a = *(const float4*)(y + row + i);
      for (int s = 1; s < slices; ++s) {
        const float4 u = *(const float4*)(y + s * slice_stride + row + i);
        a.x += u.x; a.y += u.y; a.z += u.z; a.w += u.w;
      }
      v = make_float4(__fadd_rn(v.x, a.x), __fadd_rn(v.y, a.y), __fadd_rn(v.z, a.z), __fadd_rn(v.w, a.w));
      *(float4*)(x + row + i) = v;
    }
    return v;
  };
  float4 keep[NORM_ADD_KEEP];
  float ss = 0.f;
  auto square = [&](float4 v) { ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss)))); };
  if (in_regs) {
#pragma unroll
    for (int k = 0; k < NORM_ADD_KEEP; ++k) {
      const int i = 4 * (threadIdx.x + k * NORM_ADD_THREADS);
      if (i < n) { keep[k] = fresh(i); square(keep[k]); }
    }
  } else {
    for (int i = 4 * threadIdx.x; i < n; i += 4 * NORM_ADD_THREADS) square(fresh(i));
  }
  if (!w) return;
  const float inv = inv_rms(block_sum(ss, sh), n, eps);
  auto put = [&](int i, float4 v) {
    const float4 ww = *(const float4*)(w + i);
    v = make_float4(__fmul_rn(__fmul_rn(v.x, inv), ww.x), __fmul_rn(__fmul_rn(v.y, inv), ww.y), __fmul_rn(__fmul_rn(v.z, inv), ww.z),
                    __fmul_rn(__fmul_rn(v.w, inv), ww.w));
    if (h) *(float4*)(h + row + i) = v;
    if (h16) *(uint2*)(h16 + row + i) = pack4_bf16(v);
  };
  if (in_regs) {
#pragma unroll
    for (int k = 0; k < NORM_ADD_KEEP; ++k) {
      const int i = 4 * (threadIdx.x + k * NORM_ADD_THREADS);
      if (i < n) put(i, keep[k]);
    }
  } else {
    for (int i = 4 * threadIdx.x; i < n; i += 4 * NORM_ADD_THREADS) put(i, *(const float4*)(x + row + i));  // this thread's own
  }
}

// ---- gated unit ----------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
gated_unit_kernel(const float* __restrict__ gu, GluShape sh, float* __restrict__ out, __nv_bfloat16* __restrict__ out16, int tokens) {
  pdl_enter();
  const int64_t step = (int64_t)gridDim.x * blockDim.x, first = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (sh.n % 4 == 0) {
    const int n4 = sh.n / 4;
    for (int64_t i = first; i < (int64_t)tokens * n4; i += step) {
      const int64_t t = i / n4, c = 4 * (i % n4);
      const float4 a = *(const float4*)(gu + t * 2 * sh.n + c), b = *(const float4*)(gu + t * 2 * sh.n + sh.n + c);
      const float4 r = make_float4(gated_unit(a.x, b.x, sh), gated_unit(a.y, b.y, sh), gated_unit(a.z, b.z, sh), gated_unit(a.w, b.w, sh));
      if (out) *(float4*)(out + t * sh.n + c) = r;
      if (out16) *(uint2*)(out16 + t * sh.n + c) = pack4_bf16(r);
    }
    return;
  }
  for (int64_t i = first; i < (int64_t)tokens * sh.n; i += step) {
    const int64_t t = i / sh.n, c = i % sh.n;
    const float r = gated_unit(gu[t * 2 * sh.n + c], gu[t * 2 * sh.n + sh.n + c], sh);
    if (out) out[i] = r;
    if (out16) out16[i] = __float2bfloat16_rn(r);
  }
}

// ---- launch shapes of the attention kernels ---------------------------------------------------------------------------
constexpr int MAX_VALUE = 4 * ATT_THREADS;
int span_visible(const SpanShape& sh) {
  return sh.window > 0 ? (int)std::min<int64_t>(sh.n_ctx, (int64_t)sh.window + sh.keep_first) : sh.n_ctx;
}
int span_chunk(const SpanShape& sh) { return std::max(32, (span_visible(sh) + 31) / 32); }
int span_splits(const SpanShape& sh) { return (span_visible(sh) + span_chunk(sh) - 1) / span_chunk(sh); }
size_t span_row_floats(const SpanShape& sh) {
  const size_t gq = sh.n_head / sh.n_kv, per = span_heads(sh), groups = (gq + per - 1) / per;
  return sh.n_kv * groups * span_splits(sh) * per * (size_t)(sh.dv + 2);
}
size_t span_smem(const SpanShape& sh) {
  const size_t heads = std::min(span_heads(sh), sh.n_head / sh.n_kv), P = std::max(1, ATT_THREADS / sh.dv);
  return span_chunk(sh) * sizeof(int2) + (heads * sh.dk + std::max(heads * span_chunk(sh), P * heads * sh.dv)) * sizeof(float);
}
constexpr size_t SCRATCH_FLOATS = 16u << 20;
int span_rows_per_pass(const SpanShape& sh) { return (int)std::min<size_t>(512, std::max<size_t>(1, SCRATCH_FLOATS / span_row_floats(sh))); }

// most keys a group of consecutive rows sees
int span_group_keys(const SpanShape& sh, int rows) {
  return sh.window > 0 ? (int)std::min<int64_t>(sh.n_ctx, (int64_t)sh.window + sh.keep_first + rows) : sh.n_ctx;
}
constexpr size_t MMA_SMEM_LIMIT = 222 * 1024;

typedef void (*MmaKernel)(const float*, int64_t, SpanShape, const __half*, const __half*, bool, RowMap, int, int, SpanOut);
// the smallest instantiation that covers the value dimensions
MmaKernel mma_kernel(int dv, int* nd, int* ns) {
#define LLR_SPAN(N, S) if (dv <= 8 * N * S) { *nd = N; *ns = S; return span_mma_kernel<N, S>; }
  LLR_SPAN(4, 1) LLR_SPAN(8, 1) LLR_SPAN(12, 1) LLR_SPAN(16, 1) LLR_SPAN(12, 2) LLR_SPAN(16, 2) LLR_SPAN(12, 4) LLR_SPAN(16, 4)
#undef LLR_SPAN
  return nullptr;
}

}  // namespace

cudaError_t launch_embed(const void* table, const void* pos_table, const int* ids, const RowMap& rows, float scale, float* x, void* x16,
                         int tokens, int n, const RotTable& rot, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(embed_kernel, dim3(tokens), dim3(256), 0, s, (const uint16_t*)table, (const uint16_t*)pos_table, ids, rows, scale, x,
                     (__nv_bfloat16*)x16, n, rot);
}

cudaError_t launch_qkv_store(float* proj, int ld, const float* bias, const float* q_norm, const float* k_norm, const QkvShape& sh, const RotRows& rot,
                             const RotHeads& also, const LayerKv& kv, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(qkv_store_kernel, dim3(tokens), dim3(PROJ_THREADS), 0, s, proj, ld, bias, q_norm, k_norm, sh, rot, also, kv, rows);
}

cudaError_t launch_rotate_heads(const RotHeads& h, int ld, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0 || h.heads <= 0 || h.rot.dims <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(rotate_heads_kernel, dim3(tokens), dim3(256), 0, s, h, ld);
}

cudaError_t launch_latent_store(const float* proj, int ld, const float* w, int n, float eps, const LayerKv& kv, const RowMap& rows, int tokens,
                                cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(latent_store_kernel, dim3(tokens), dim3(PROJ_THREADS), 0, s, proj, ld, w, n, eps, kv, rows);
}

cudaError_t launch_rows_bf16(const float* x, int64_t ld, int n, void* out16, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(rows_bf16_kernel, dim3(tokens), dim3(256), 0, s, x, ld, n, (__nv_bfloat16*)out16);
}

cudaError_t launch_head_product_t(const void* w, int heads, int rows, int cols, const float* x, int64_t x_ld, float* y, int tokens, cudaStream_t s,
                                  uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  if (tokens == 1)
    return launch_walk(head_product_t_kernel<1>, dim3((cols + 127) / 128, heads, 1), dim3(256), 0, s, (const uint16_t*)w, heads, rows, cols, x, x_ld, y, tokens);
  return launch_walk(head_product_t_kernel<8>, dim3((cols + 127) / 128, heads, (tokens + 7) / 8), dim3(256), 0, s, (const uint16_t*)w, heads, rows, cols, x,
                     x_ld, y, tokens);
}

cudaError_t launch_head_product(const void* w, int heads, int rows, int cols, const float* x, int64_t x_ld, float* y, const float* gate,
                                int64_t gate_ld, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  if (tokens == 1)
    return launch_walk(head_product_kernel<1>, dim3((heads * rows + 7) / 8, 1), dim3(256), 0, s, (const uint16_t*)w, heads, rows, cols, x, x_ld, y, gate,
                       gate_ld, tokens);
  return launch_walk(head_product_kernel<8>, dim3((heads * rows + 7) / 8, (tokens + 7) / 8), dim3(256), 0, s, (const uint16_t*)w, heads, rows, cols, x, x_ld,
                     y, gate, gate_ld, tokens);
}

cudaError_t launch_head_transpose(const void* w, int heads, int rows, int cols, void* out, cudaStream_t s, uint64_t* launches) {
  if (launches) ++*launches;
  head_transpose_kernel<<<dim3((unsigned)std::min<int64_t>(((int64_t)rows * cols + 255) / 256, 256), heads), 256, 0, s>>>((const uint16_t*)w, rows, cols,
                                                                                                                     (uint16_t*)out);
  return cudaGetLastError();
}

bool span_supported(const SpanShape& sh) {
  return sh.n_head > 0 && sh.n_kv > 0 && sh.n_head % sh.n_kv == 0 && sh.dk > 0 && sh.dv > 0 && sh.dv <= MAX_VALUE && sh.dk <= 1024 && sh.n_head <= 4096 &&
         span_smem(sh) <= 200 * 1024;
}
size_t span_scratch_floats(const SpanShape& sh, int max_rows) {
  int nd = 0, ns = 0;
  size_t gathered = 0;  // binary16 keys and values of one group
  if (mma_kernel(sh.dv, &nd, &ns)) {
    const MmaLayout L = mma_layout(sh.dk, sh.dv, nd, ns, false);  // not shared: the larger of the two
    gathered = (size_t)sh.n_kv * span_group_keys(sh, max_rows) * (L.kr + L.vr) / 2 + 64;
  }
  return std::max((size_t)span_rows_per_pass(sh) * span_row_floats(sh), gathered);
}

cudaError_t launch_span_attention(const float* q, int64_t q_ld, const SpanShape& sh, const LayerKv& kv, const RowMap& rows, int t0, int tokens,
                                  const SpanOut& out, float* scratch, bool tensor_cores, bool one_sequence, const NewToken* nt, cudaStream_t s,
                                  uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (!span_supported(sh)) return cudaErrorInvalidValue;
  const int gq = sh.n_head / sh.n_kv;
  if (tensor_cores && one_sequence && sh.dk % 8 == 0 && sh.dv % 8 == 0 && out.ld % 2 == 0 && ((uintptr_t)out.out & 7) == 0 && ((uintptr_t)out.out16 & 3) == 0 &&
      (!out.gate || out.head_gate || (out.gate_ld % 2 == 0 && ((uintptr_t)out.gate & 7) == 0))) {
    int nd = 0, ns = 0;
    MmaKernel kern = mma_kernel(sh.dv, &nd, &ns);
    const bool shared = kv.k == kv.v;
    const MmaLayout L = mma_layout(sh.dk, sh.dv, nd, ns, shared);
    const size_t smem = kern ? mma_smem(L, ns) : 0;
    if (kern && smem <= MMA_SMEM_LIMIT) {
      if (smem > 40 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute((const void*)kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
      }
      if (launches) *launches += 2;
      const int keys = span_group_keys(sh, tokens);
      __half* k16 = (__half*)scratch;
      __half* v16 = shared ? k16 : k16 + (size_t)sh.n_kv * keys * L.kr;
      cudaError_t e = launch_walk(span_gather_kernel, dim3((keys + 7) / 8, sh.n_kv), dim3(256), 0, s, sh, kv, rows, t0, tokens, L.kr, L.vr, k16, v16);
      if (e != cudaSuccess) return e;
      return launch_walk(kern, dim3((unsigned)(((int64_t)tokens * gq + 63) / 64), sh.n_kv), dim3(128 * ns), smem, s, q, q_ld, sh, (const __half*)k16,
                         (const __half*)v16, shared, rows, t0, tokens, out);
    }
  }
  const int groups = (gq + span_heads(sh) - 1) / span_heads(sh), chunk = span_chunk(sh), splits = span_splits(sh), per = span_rows_per_pass(sh);
  const size_t smem = span_smem(sh);
  auto kern = sh.dv <= ATT_THREADS ? span_partial_kernel<ATT_THREADS> : sh.dv <= 2 * ATT_THREADS ? span_partial_kernel<2 * ATT_THREADS> : span_partial_kernel<MAX_VALUE>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute((const void*)kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  for (int r = 0; r < tokens; r += per) {
    const int n = std::min(per, tokens - r);
    if (launches) *launches += 2;
    cudaError_t e = launch_walk(kern, dim3(sh.n_kv * groups, splits, n), dim3(ATT_THREADS), smem, s, q, q_ld, sh, kv, rows, t0 + r, chunk, scratch,
                                nt && tokens == 1 ? *nt : NewToken{});
    if (e != cudaSuccess) return e;
    e = launch_walk(span_combine_kernel, dim3(sh.n_head, n, (sh.dv + 127) / 128), dim3(128), 0, s, (const float*)scratch, sh, rows, t0 + r, splits, out);
    if (e != cudaSuccess) return e;
  }
  return cudaSuccess;
}

cudaError_t launch_norm_add(float* x, const float* y, int slices, int64_t slice_stride, const float* w, float eps, void* x16, int tokens, int n,
                            cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(norm_add_kernel, dim3(tokens), dim3(NORM_ADD_THREADS), 0, s, x, y, slices, slice_stride, w, eps, (__nv_bfloat16*)x16, n);
}

cudaError_t launch_add_norm(float* x, const float* y, int slices, int64_t slice_stride, const float* w, float eps, float* h, void* h16, int tokens,
                            int n, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (n % 4 != 0) return cudaErrorInvalidValue;
  if (launches) ++*launches;
  return launch_walk(add_norm_kernel, dim3(tokens), dim3(NORM_ADD_THREADS), 0, s, x, y, slices, slice_stride, w, eps, h, (__nv_bfloat16*)h16, n);
}

cudaError_t launch_gated_unit(const float* gu, const GluShape& sh, float* out, void* out16, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  const int64_t n = (int64_t)tokens * sh.n / (sh.n % 4 == 0 ? 4 : 1);
  return launch_walk(gated_unit_kernel, dim3((unsigned)std::max<int64_t>(1, std::min<int64_t>((n + 255) / 256, 148 * 8))), dim3(256), 0, s, gu, sh, out,
                     (__nv_bfloat16*)out16, tokens);
}

}  // namespace llr
