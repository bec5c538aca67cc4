// Recurrent mixers of decoders described layer by layer: a state per sequence that every token fades and adds to, instead of
// cached positions.
//   (a) matrix states per head: retention (a fixed decay per head) and the gated delta rule (a decay per head and key channel,
//       a correction of what the state holds for the key),
//   (b) a real-gated linear recurrence per channel,
//   (c) the short causal convolutions in front of them, whose last inputs belong to the state.
//
// Every recurrence runs token by token in f32 from state kept in registers: the result of a position has the same bits however
// its prompt was cut.  What makes that fast on this machine is width instead of depth -- a column of a matrix state depends on
// no other column, a channel on no other channel -- and that a step's only dependent chain is one reduction (delta rule) or
// one multiply-add (the others): inputs of the next tokens arrive in shared memory by asynchronous copies meanwhile, and the
// convolutions, unit vectors, decays and gates of all tokens are computed in parallel before the scan.
//
// A sequence whose first row stands at position 0 starts from zeros: a slot that is used again needs no clearing.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>

#include "llr_attend.cuh"
#include "llr_kernels.cuh"

namespace llr {
namespace {

__device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return z > 0.f ? z + log1pf(expf(-z)) : log1pf(expf(z)); }

struct Group { int t0, t1, seq; bool fresh; };
__device__ __forceinline__ Group group_of(const RowGroups& g, const RowMap& rows, int tokens, int i) {
  const int t0 = g.first ? g.first[i] : 0, t1 = g.first ? g.first[i + 1] : tokens;
  return Group{t0, t1, row_sequence(rows, t0), row_position(rows, t0) == 0};
}

// ---- short convolution ------------------------------------------------------------------------------------------------
// How many of the `back` rows before row t belong to its sequence and stand in this batch
__device__ __forceinline__ int rows_before(const RowMap& rows, int t, int back) {
  if (!rows.row_seq) return min(t, back);
  int n = 0;
  while (n < back && t - n - 1 >= 0 && rows.row_seq[t - n - 1] == rows.row_seq[t]) ++n;
  return n;
}
// channel c at row t; near: rows_before(t, taps - 1), pos: the row's position.  Oldest input first.
__device__ __forceinline__ float conv_at(const float* x, int64_t ld, const ConvShape& cv, const float* tail, int t, int near, int pos, int c) {
  const float b = cv.bias ? cv.bias[c] : 0.f;
  float acc = 0.f;
#pragma unroll 4
  for (int j = cv.taps - 1; j >= 0; --j) {
    float v = 0.f;
    if (j <= near) v = __fadd_rn(x[(int64_t)(t - j) * ld + c], b);
    else if (j <= pos) v = tail[(int64_t)(cv.taps - 1 - (j - near)) * cv.channels + c];
    acc = fmaf(cv.w[(int64_t)(cv.taps - 1 - j) * cv.channels + c], v, acc);
  }
  return cv.out_bias ? __fadd_rn(acc, cv.out_bias[c]) : acc;
}
// channels c .. c + 3, all on 16-byte boundaries: the same sums
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(__fadd_rn(a.x, b.x), __fadd_rn(a.y, b.y), __fadd_rn(a.z, b.z), __fadd_rn(a.w, b.w)); }
__device__ __forceinline__ float4 conv4_at(const float* x, int64_t ld, const ConvShape& cv, const float* tail, int t, int near, int pos, int c) {
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 b = cv.bias ? *(const float4*)(cv.bias + c) : acc;
#pragma unroll 4
  for (int j = cv.taps - 1; j >= 0; --j) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j <= near) {
      v = *(const float4*)(x + (int64_t)(t - j) * ld + c);
      if (cv.bias) v = add4(v, b);
    }
    else if (j <= pos) {
      v = *(const float4*)(tail + (int64_t)(cv.taps - 1 - (j - near)) * cv.channels + c);
    }
    const float4 w = *(const float4*)(cv.w + (int64_t)(cv.taps - 1 - j) * cv.channels + c);
    acc = make_float4(fmaf(w.x, v.x, acc.x), fmaf(w.y, v.y, acc.y), fmaf(w.z, v.z, acc.z), fmaf(w.w, v.w, acc.w));
  }
  return cv.out_bias ? add4(acc, *(const float4*)(cv.out_bias + c)) : acc;
}
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + expf(-z)); }
__device__ __forceinline__ float4 silu4(float4 z) { return make_float4(silu(z.x), silu(z.y), silu(z.z), silu(z.w)); }
// The last taps - 1 inputs behind the group's rows become the state's; thread `at` of `all` owns every all-th channel.
__device__ __forceinline__ void conv_tail_update(const float* x, int64_t ld, const ConvShape& cv, const Group& g, int at, int all) {
  if (cv.taps < 2) return;
  float* tail = cv.tail.state + g.seq * cv.tail.stride;
  const int keep = cv.taps - 1, n = g.t1 - g.t0;
  for (int c = at; c < cv.channels; c += all) {
    const float b = cv.bias ? cv.bias[c] : 0.f;
    for (int k0 = 0; k0 < keep; k0 += 4) {  // ascending: what moves down is read before it is written
      float v[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int k = k0 + j, back = keep - k;  // rows before the next one
        v[j] = 0.f;
        if (k < keep) {
          if (back <= n) v[j] = __fadd_rn(x[(int64_t)(g.t1 - back) * ld + c], b);
          else if (!g.fresh) v[j] = tail[(int64_t)(k + n) * cv.channels + c];
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (k0 + j < keep) tail[(int64_t)(k0 + j) * cv.channels + c] = v[j];
    }
  }
}

// v as a sum of three bfloat16 values: 24 bits of mantissa
__device__ __forceinline__ void in_parts(float v, __nv_bfloat16 (&p)[3]) {
  p[0] = __float2bfloat16_rn(v);
  v = __fsub_rn(v, __bfloat162float(p[0]));
  p[1] = __float2bfloat16_rn(v);
  p[2] = __float2bfloat16_rn(__fsub_rn(v, __bfloat162float(p[1])));
}
// grid (row, CONV_COLS channels); vec: four channels per thread, everything on boundaries of four
constexpr int CONV_THREADS = 128;
__global__ void __launch_bounds__(CONV_THREADS)
conv_rows_kernel(const float* __restrict__ x, int64_t ld, ConvShape cv, float* __restrict__ u, __nv_bfloat16* __restrict__ u16, int block, RowMap rows, bool vec) {
  pdl_enter();
  const int t = blockIdx.x, near = rows_before(rows, t, cv.taps - 1), pos = row_position(rows, t), at = blockIdx.y * CONV_THREADS + threadIdx.x;
  const float* tail = cv.tail.state + row_sequence(rows, t) * cv.tail.stride;
  if (vec) {
    const int c = 4 * at;
    if (c >= cv.channels) return;
    const float4 v = conv4_at(x, ld, cv, tail, t, near, pos, c);
    *(float4*)(u + (int64_t)t * cv.channels + c) = v;
    if (u16) {
      __nv_bfloat16 p[4][3];
      in_parts(v.x, p[0]); in_parts(v.y, p[1]); in_parts(v.z, p[2]); in_parts(v.w, p[3]);
      __nv_bfloat16* o = u16 + (int64_t)t * 3 * cv.channels + (int64_t)(c / block) * 3 * block + c % block;
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        const __nv_bfloat162 lo = __halves2bfloat162(p[0][k], p[1][k]), hi = __halves2bfloat162(p[2][k], p[3][k]);
        *(uint2*)(o + k * block) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
      }
    }
    return;
  }
  if (at >= cv.channels) return;
  const float v = conv_at(x, ld, cv, tail, t, near, pos, at);
  u[(int64_t)t * cv.channels + at] = v;
  if (u16) {
    __nv_bfloat16 p[3];
    in_parts(v, p);
    __nv_bfloat16* o = u16 + (int64_t)t * 3 * cv.channels + (int64_t)(at / block) * 3 * block + at % block;
#pragma unroll
    for (int k = 0; k < 3; ++k) o[k * block] = p[k];
  }
}

__global__ void triple_columns_kernel(const uint16_t* __restrict__ w, int64_t n, int cols, uint16_t* __restrict__ out) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t at = i / cols * 3 * cols + i % cols;
    out[at] = out[at + cols] = out[at + 2 * cols] = w[i];
  }
}

// ---- inputs of the delta rule -------------------------------------------------------------------------------------------
__device__ __forceinline__ float fade(float rate, float a, float bias) { return expf(-__fmul_rn(rate, softplus(__fadd_rn(a, bias)))); }

// grid (row, key/value head), a thread per value where they fit a block: the head's query and key, and values and decays of the
// heads that share them
__global__ void __launch_bounds__(1024)
delta_prepare_kernel(const float* __restrict__ proj, int64_t ld, const float* __restrict__ a, const float* __restrict__ b, DeltaShape d, ConvShape cv,
                     float* __restrict__ prep, int64_t prep_ld, RowMap rows) {
  pdl_enter();
  extern __shared__ float qk[];  // the head's q | k behind convolution and silu
  __shared__ float red[3][32];
  const int t = blockIdx.x, kvh = blockIdx.y, near = rows_before(rows, t, cv.taps - 1), pos = row_position(rows, t), share = d.n_head / d.n_kv;
  const float* tail = cv.tail.state + row_sequence(rows, t) * cv.tail.stride;
  const int nq = d.n_kv * d.dim, nv = d.n_head * d.vdim, ng = d.n_head * d.dim;
  const int end_v = 2 * d.dim + share * d.vdim, end = end_v + share * d.dim;
  float* o = prep + (int64_t)t * prep_ld;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < end; i += blockDim.x) {
    if (i < end_v) {
      const int c = i < d.dim ? kvh * d.dim + i : i < 2 * d.dim ? nq + kvh * d.dim + i - d.dim : 2 * nq + kvh * share * d.vdim + i - 2 * d.dim;
      const float v = silu(conv_at(proj, ld, cv, tail, t, near, pos, c));
      if (i < 2 * d.dim) qk[i] = v;
      else o[c] = v;
      if (i < d.dim) sq = fmaf(v, v, sq);
      else if (i < 2 * d.dim) sk = fmaf(v, v, sk);
    } else {
      const int c = kvh * share * d.dim + i - end_v;
      o[2 * nq + nv + c] = fade(d.rate[c / d.dim], a[(int64_t)t * ng + c], d.step_bias[c]);
    }
  }
  for (int j = threadIdx.x; j < share; j += blockDim.x) o[2 * nq + nv + ng + kvh * share + j] = sigmoid(b[(int64_t)t * ld + kvh * share + j]);
  sq = sqrtf(__fadd_rn(block_sum(sq, red[0]), d.unit_eps));
  sk = sqrtf(__fadd_rn(block_sum(sk, red[1]), d.unit_eps));
  float kq = 0.f;
  for (int i = threadIdx.x; i < d.dim; i += blockDim.x) {  // qk is complete: the sums have synchronized
    const float qv = __fmul_rn(__fdiv_rn(qk[i], sq), d.q_scale), kv = __fdiv_rn(qk[d.dim + i], sk);
    o[kvh * d.dim + i] = qv;
    o[nq + kvh * d.dim + i] = kv;
    kq = fmaf(kv, qv, kq);
  }
  kq = block_sum(kq, red[2]);
  if (threadIdx.x == 0) o[2 * nq + nv + ng + d.n_head + kvh] = kq;
}

// ---- four rows at a time ------------------------------------------------------------------------------------------------
// Rows 1 .. 4 of a block, with P_i = g_1 .. g_i per key channel, read the state S before the block:
//   S_i = diag(P_i) S + sum_(j <= i) diag(g_(j+1) .. g_i) k_j u_j^T,
//   u_i = beta_i (v_i - S^T (P_i k_i) - sum_(j < i) c_ij u_j),   c_ij = k_i^T diag(g_(j+1) .. g_i) k_j,
//   o_i = S^T (P_i q_i) + sum_(j <= i) s_ij u_j,                 s_ij = q_i^T diag(g_(j+1) .. g_i) k_j,
// so a block has one chain of reductions where its rows had four, and nothing is divided by a decay.  A record per block and
// head holds the vectors [DP each]
//   delta rule: P_i k_i | P_i q_i | g_(i+1) .. g_4 k_i | P_4, retention (decay a, u_i = v_i): a^i q_i | a^(4-i) k_i,
// then s [4][4], c [4][4], beta [4], and a^(rows of the block).  Rows behind the group's end have k = q = 0 and fade nothing.
constexpr int BLOCK_ROWS = 4, REC_SCALARS = 40;
__host__ __device__ constexpr int rec_vectors(bool delta) { return delta ? 13 : 8; }
__host__ __device__ constexpr int rec_floats(int dp, bool delta) { return rec_vectors(delta) * dp + REC_SCALARS; }
inline int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : 128; }
// Group i's first block; its blocks follow each other, and groups do not overlap.
__device__ __forceinline__ int first_block(const RowGroups& g, int i) { return (g.first ? g.first[i] : 0) / BLOCK_ROWS + i; }
struct BlockAt { int t0, n; };  // first row, rows (0: no such block)
__device__ __forceinline__ BlockAt block_at(const RowGroups& g, int tokens, int slot) {
  int lo = 0, hi = g.n - 1;
  while (lo < hi) {  // the last group that starts at slot or before it
    const int mid = (lo + hi + 1) / 2;
    if (first_block(g, mid) <= slot) lo = mid;
    else hi = mid - 1;
  }
  const int t0 = g.first ? g.first[lo] : 0, t1 = g.first ? g.first[lo + 1] : tokens, t = t0 + BLOCK_ROWS * (slot - first_block(g, lo));
  return BlockAt{t, min(BLOCK_ROWS, t1 - t)};
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 mul4(float4 a, float b) { return make_float4(a.x * b, a.y * b, a.z * b, a.w * b); }
__device__ __forceinline__ float dot4(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }

// grid (block of rows, head), a warp per row, a lane per four key channels
__global__ void __launch_bounds__(32 * BLOCK_ROWS)
delta_blocks_kernel(const float* __restrict__ proj, int64_t ld, const float* __restrict__ a, const float* __restrict__ b, DeltaShape d, ConvShape cv,
                    int dp, float* __restrict__ rec, float* __restrict__ v_out, RowGroups groups, RowMap rows, int tokens) {
  pdl_enter();
  __shared__ float4 sq[BLOCK_ROWS][32], sk[BLOCK_ROWS][32], sg[BLOCK_ROWS][32];
  const int lane = threadIdx.x & 31, i = threadIdx.x >> 5, slot = blockIdx.x, h = blockIdx.y, kvh = h / (d.n_head / d.n_kv);
  const BlockAt at = block_at(groups, tokens, slot);
  if (at.n <= 0) return;
  const int nq = d.n_kv * d.dim, nv = d.n_head * d.vdim, ng = d.n_head * d.dim, c = 4 * lane, t = at.t0 + i;
  float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q, g = make_float4(1.f, 1.f, 1.f, 1.f);
  float* o = rec + ((int64_t)slot * d.n_head + h) * rec_floats(dp, true);
  float* sc = o + rec_vectors(true) * dp;
  if (i < at.n) {
    const int near = rows_before(rows, t, cv.taps - 1), pos = row_position(rows, t);
    const float* tail = cv.tail.state + row_sequence(rows, t) * cv.tail.stride;
    if (c < d.dim) {
      const float rate = d.rate[h];
      const float4 s = *(const float4*)(a + (int64_t)t * ng + h * d.dim + c), bias = *(const float4*)(d.step_bias + h * d.dim + c);
      q = silu4(conv4_at(proj, ld, cv, tail, t, near, pos, kvh * d.dim + c));
      k = silu4(conv4_at(proj, ld, cv, tail, t, near, pos, nq + kvh * d.dim + c));
      g = make_float4(fade(rate, s.x, bias.x), fade(rate, s.y, bias.y), fade(rate, s.z, bias.z), fade(rate, s.w, bias.w));
    }
    for (int j = c; j < d.vdim; j += 128)
      *(float4*)(v_out + (int64_t)t * nv + h * d.vdim + j) = silu4(conv4_at(proj, ld, cv, tail, t, near, pos, 2 * nq + h * d.vdim + j));
    q = mul4(q, __fdiv_rn(d.q_scale, sqrtf(__fadd_rn(warp_sum(dot4(q, q)), d.unit_eps))));
    k = mul4(k, __fdiv_rn(1.0f, sqrtf(__fadd_rn(warp_sum(dot4(k, k)), d.unit_eps))));
  }
  sq[i][lane] = q;
  sk[i][lane] = k;
  sg[i][lane] = g;
  if (lane == 0) sc[32 + i] = i < at.n ? sigmoid(b[(int64_t)t * ld + h]) : 0.f;
  __syncthreads();
  // row i against the rows up to it: k_j faded from j to i, the last j first
  float4 f = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
  for (int j = BLOCK_ROWS - 1; j >= 0; --j) {
    float sij = 0.f, cij = 0.f;
    if (j <= i) {
      const float4 kj = mul4(f, sk[j][lane]);
      sij = warp_sum(dot4(kj, q));
      if (j < i) cij = warp_sum(dot4(kj, k));
      f = mul4(f, sg[j][lane]);
    }
    if (lane == 0) { sc[4 * i + j] = sij; sc[16 + 4 * i + j] = cij; }
  }
  // f: all decays up to row i; the decays behind it
  float4 after = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
  for (int j = 1; j < BLOCK_ROWS; ++j)
    if (j > i) after = mul4(after, sg[j][lane]);
  auto put = [&](int at, float4 v) { if (c < dp) *(float4*)(o + at * dp + c) = v; };
  put(i, mul4(f, k));
  put(BLOCK_ROWS + i, mul4(f, q));
  put(2 * BLOCK_ROWS + i, mul4(after, k));
  if (i == BLOCK_ROWS - 1) put(3 * BLOCK_ROWS, f);
}

// the same for retention, from rotated queries and keys
__global__ void __launch_bounds__(128)
retention_blocks_kernel(MatrixScan m, int dp, float* __restrict__ rec, RowGroups groups, int tokens, int slots) {
  pdl_enter();
  const int lane = threadIdx.x & 31, w = blockIdx.x * 4 + (threadIdx.x >> 5), slot = w / m.n_head, h = w % m.n_head, kvh = h / (m.n_head / m.n_kv);
  if (slot >= slots) return;
  const BlockAt at = block_at(groups, tokens, slot);
  if (at.n <= 0) return;
  const int c = 4 * lane;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const float decay = m.decay[h];
  float pw[5];
  pw[0] = 1.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) pw[i + 1] = pw[i] * decay;
  float4 q[4], k[4];
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const bool on = r < at.n && c < m.dim;
    const int64_t row = (int64_t)(at.t0 + r) * m.ld + (int64_t)kvh * m.dim + c;
    q[r] = on ? *(const float4*)(m.q + row) : zero;
    k[r] = on ? mul4(*(const float4*)(m.k + row), m.k_scale) : zero;
  }
  float* o = rec + ((int64_t)slot * m.n_head + h) * rec_floats(dp, false);
  float* sc = o + rec_vectors(false) * dp;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float after = i < at.n ? (at.n == 4 ? pw[3 - i] : at.n == 3 ? (i < 3 ? pw[i < 3 ? 2 - i : 0] : 0.f) : at.n == 2 ? pw[i < 2 ? 1 - i : 0] : pw[0]) : 0.f;
    if (c < dp) {
      *(float4*)(o + i * dp + c) = mul4(q[i], pw[i + 1]);
      *(float4*)(o + (4 + i) * dp + c) = mul4(k[i], after);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float s = j <= i ? warp_sum(dot4(q[i], k[j])) * pw[i >= j ? i - j : 0] : 0.f;
      if (lane == 0) sc[4 * i + j] = s;
    }
  }
  if (lane == 0) sc[36] = at.n == 4 ? pw[4] : at.n == 3 ? pw[3] : at.n == 2 ? pw[2] : pw[1];
}

// ---- matrix states --------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// a head's result behind its norm and gate; a warp per head and row
__device__ __forceinline__ void head_out(const float* o, int vdim, const HeadOut& ho, int t, int h, int lane) {
  const float* gate = ho.gate + (int64_t)t * ho.gate_ld + (int64_t)h * vdim;
  const int64_t at = (int64_t)t * ho.ld + (int64_t)h * vdim;
  auto inverse = [&](float ss) { return __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(warp_sum(ss), (float)vdim), ho.eps))); };
  auto value = [&](float v, float inv, int i, float g) {
    v = __fmul_rn(v, inv);
    if (ho.weight) v = __fmul_rn(v, ho.weight[i]);
    return __fmul_rn(__fmul_rn(v, ho.silu ? __fmul_rn(g, sigmoid(g)) : sigmoid(g)), ho.scale);
  };
  __nv_bfloat16* out16 = (__nv_bfloat16*)ho.out16;
  const bool vec = (vdim & 3) == 0 && vdim <= 256 && (((uintptr_t)o | (uintptr_t)gate) & 15) == 0 && (!ho.out || ((uintptr_t)(ho.out + at) & 15) == 0) &&
                   (!out16 || ((uintptr_t)(out16 + at) & 7) == 0);
  if (vec) {  // the whole head at once
    float4 v[2], g[2];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = 4 * (lane + 32 * j);
      if (i < vdim) {
        v[j] = *(const float4*)(o + i);
        g[j] = *(const float4*)(gate + i);
        ss = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, ss))));
      }
    }
    const float inv = inverse(ss);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = 4 * (lane + 32 * j);
      if (i < vdim) {
        const float4 r = make_float4(value(v[j].x, inv, i, g[j].x), value(v[j].y, inv, i + 1, g[j].y), value(v[j].z, inv, i + 2, g[j].z),
                                     value(v[j].w, inv, i + 3, g[j].w));
        if (ho.out) *(float4*)(ho.out + at + i) = r;
        if (out16) {
          const __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
          *(uint2*)(out16 + at + i) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
        }
      }
    }
    return;
  }
  float ss = 0.f;
  for (int i = lane; i < vdim; i += 32) ss = fmaf(o[i], o[i], ss);
  const float inv = inverse(ss);
  for (int i = lane; i < vdim; i += 32) {
    const float v = value(o[i], inv, i, gate[i]);
    if (ho.out) ho.out[at + i] = v;
    if (out16) out16[at + i] = __float2bfloat16_rn(v);
  }
}
__global__ void __launch_bounds__(256)
head_out_kernel(const float* __restrict__ o, int heads, int vdim, HeadOut ho, int tokens) {
  pdl_enter();
  const int64_t i = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= (int64_t)tokens * heads) return;
  head_out(o + i * vdim, vdim, ho, (int)(i / heads), (int)(i % heads), threadIdx.x & 31);
}

// Pairs of f32 values in one register pair: two multiply-adds per instruction, each rounded as fmaf rounds
typedef unsigned long long pair;
__device__ __forceinline__ pair fma2(pair a, pair b, pair c) {
  pair d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ pair mul2(pair a, pair b) {
  pair d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ pair both(float v) { return (pair)__float_as_uint(v) << 32 | __float_as_uint(v); }
__device__ __forceinline__ pair make_pair(float lo, float hi) { return (pair)__float_as_uint(hi) << 32 | __float_as_uint(lo); }
__device__ __forceinline__ float low(pair p) { return __uint_as_float((uint32_t)p); }
__device__ __forceinline__ float high(pair p) { return __uint_as_float((uint32_t)(p >> 32)); }

constexpr int SCAN_STAGES = 3;  // stages in flight
// Shared memory of a block, in floats: per stage q | k (| g) of DP values per row, v and one pair (beta, k . q) per row
template <int DP, bool DELTA>
struct ScanLay {
  static constexpr int VEC = DP * (DELTA ? 3 : 2), ROWS = DP > 256 ? 2 : 8;  // rows per stage
  static __host__ __device__ int stage(int cols) { return ROWS * (VEC + ((cols + 3) & ~3) + 4); }
  static __host__ __device__ int total(int cols) { return SCAN_STAGES * stage(cols); }
};
constexpr int scan_threads(int r) { return r > 16 ? 256 : 512; }  // most threads of a block: the state stays in registers

// grid (column group, head, group of rows); cols / C * LPC threads.  LPC lanes hold C columns: lane l the values 4 (l + LPC j) + c.
template <int LPC, int R, int C, bool DELTA>
__global__ void __launch_bounds__(scan_threads(R))
matrix_scan_kernel(MatrixScan m, HeadOut ho, RowGroups groups, RowMap rows, int tokens, int cols, bool whole, float* o_raw) {
  pdl_enter();
  constexpr int DP = LPC * R, P = R / 2;  // padded length, pairs per lane
  using L = ScanLay<DP, DELTA>;
  constexpr int ROWS = L::ROWS;
  extern __shared__ __align__(16) float sm[];
  const Group g = group_of(groups, rows, tokens, blockIdx.z);
  const int tid = threadIdx.x, nt = blockDim.x, l = tid % LPC, col = tid / LPC * C, head = blockIdx.y, kvh = head / (m.n_head / m.n_kv);
  const int c0 = blockIdx.x * cols, live = min(cols, m.vdim - c0), stage = L::stage(cols), v_ld = (cols + 3) & ~3;
  if (m.dim < DP) {  // values behind dim stay zero
    for (int i = tid; i < SCAN_STAGES * stage; i += nt) sm[i] = 0.f;
    __syncthreads();
  }
  const bool vec = ((m.dim | (int)m.ld) & 3) == 0 && (((uintptr_t)m.q | (uintptr_t)m.k | (DELTA ? (uintptr_t)m.g : 0)) & 15) == 0;
  const float *q_row = m.q + (int64_t)kvh * m.dim, *k_row = m.k + (int64_t)kvh * m.dim, *g_row = DELTA ? m.g + (int64_t)head * m.dim : nullptr,
              *v_row = m.v + (int64_t)head * m.vdim + c0;
  const int n = g.t1 - g.t0, steps = (n + ROWS - 1) / ROWS;
  auto fetch = [&](int s) {
    float* base = sm + (s % SCAN_STAGES) * stage;
    const int64_t r0 = g.t0 + s * ROWS;
    const int nr = min(ROWS, n - s * ROWS);
    auto run = [&](float* dst, const float* src) {  // nr rows of dim values, DP apart
      src += r0 * m.ld;
      if (vec) {
        for (int i = tid; i < nr * (DP / 4); i += nt) {
          const int r = i / (DP / 4), c = 4 * (i % (DP / 4));
          if (c < m.dim) async16(dst + r * DP + c, src + r * m.ld + c);
        }
      } else {
        for (int i = tid; i < nr * DP; i += nt)
          if (i % DP < m.dim) async4(dst + i, src + i / DP * m.ld + i % DP);
      }
    };
    if (m.rot.dims > 0) {  // a single row as the product left it
      const int half = m.rot.dims / 2;
      for (int i = tid; i < 2 * m.dim; i += nt) {
        const bool key = i >= m.dim;
        const int c = key ? i - m.dim : i;
        const float* src = (key ? k_row : q_row) + r0 * m.ld;
        float v = src[c];
        if (c < 2 * half) {
          const float2 a = m.rot.cs[r0 * m.rot.ld + (c < half ? c : c - half)];
          v = c < half ? fmaf(v, a.x, -__fmul_rn(src[c + half], a.y)) : fmaf(v, a.x, __fmul_rn(src[c - half], a.y));
        }
        base[(key ? ROWS * DP : 0) + c] = v;
      }
    } else {
      run(base, q_row);
      run(base + ROWS * DP, k_row);
    }
    if (DELTA) run(base + 2 * ROWS * DP, g_row);
    float* sv = base + ROWS * L::VEC;
    for (int i = tid; i < nr * cols; i += nt) {
      const int r = i / cols, c = i - r * cols;
      if (c < live) async4(sv + r * v_ld + c, v_row + (r0 + r) * m.v_ld + c);
    }
    if (DELTA && tid < nr) {
      async4(sv + ROWS * v_ld + 2 * tid, m.beta + (r0 + tid) * m.ld + head);
      async4(sv + ROWS * v_ld + 2 * tid + 1, m.kq + (r0 + tid) * m.ld + kvh);
    }
    async_commit();
  };
#pragma unroll
  for (int s = 0; s < SCAN_STAGES - 1; ++s) {
    if (s < steps) fetch(s);
    else async_commit();
  }
  // the columns' states
  float* st = m.state.state + g.seq * m.state.stride + ((int64_t)head * m.vdim + c0 + col) * m.dim;
  const bool st_vec = (m.dim & 3) == 0 && ((uintptr_t)st & 15) == 0;
  pair S[C][P];
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int j = 0; j < P; j += 2) {
      const int i = 4 * (l + LPC * (j / 2));
      const float* p = st + c * m.dim;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (col + c < live && !g.fresh) {
        if (st_vec) {
          if (i < m.dim) v = *(const float4*)(p + i);
        } else {
          if (i < m.dim) v.x = p[i];
          if (i + 1 < m.dim) v.y = p[i + 1];
          if (i + 2 < m.dim) v.z = p[i + 2];
          if (i + 3 < m.dim) v.w = p[i + 3];
        }
      }
      S[c][j] = make_pair(v.x, v.y);
      S[c][j + 1] = make_pair(v.z, v.w);
    }
  if (DELTA) conv_tail_update(m.conv_in, m.conv_ld, m.conv, g, (blockIdx.y * gridDim.x + blockIdx.x) * nt + tid, (int)(gridDim.x * gridDim.y) * nt);
  const pair decay = DELTA ? 0 : both(m.decay[head]);
  float* o_row = o_raw + ((int64_t)g.t0 * m.n_head + head) * m.vdim + c0 + col;
  const int64_t o_ld = (int64_t)m.n_head * m.vdim;
  for (int s = 0; s < steps; ++s) {
    async_wait<SCAN_STAGES - 2>();
    __syncthreads();  // stage s has arrived for every thread, and everyone is done with stage s - 1
    if (s + SCAN_STAGES - 1 < steps) fetch(s + SCAN_STAGES - 1);
    else async_commit();
    const float* base = sm + (s % SCAN_STAGES) * stage;
    const float* sv = base + ROWS * L::VEC;
    const int nr = min(ROWS, n - s * ROWS);
#pragma unroll (R <= 16 ? 2 : 1)
    for (int r = 0; r < nr; ++r, o_row += o_ld) {
      const ulonglong2* q4 = (const ulonglong2*)(base + r * DP) + l;
      const ulonglong2* k4 = (const ulonglong2*)(base + (ROWS + r) * DP) + l;
      float v[C], o[C];
#pragma unroll
      for (int c = 0; c < C; ++c) v[c] = sv[r * v_ld + col + c];
      pair acc[C][2];
#pragma unroll
      for (int c = 0; c < C; ++c) acc[c][0] = acc[c][1] = 0;
      if constexpr (DELTA) {
        const ulonglong2* g4 = (const ulonglong2*)(base + (2 * ROWS + r) * DP) + l;
        const float beta = sv[ROWS * v_ld + 2 * r], kq = sv[ROWS * v_ld + 2 * r + 1];
        pair held[C][2], kk[P];
#pragma unroll
        for (int c = 0; c < C; ++c) held[c][0] = held[c][1] = 0;
#pragma unroll
        for (int j = 0; j < P; j += 2) {
          const ulonglong2 gg = g4[LPC * (j / 2)], kj = k4[LPC * (j / 2)], qq = q4[LPC * (j / 2)];
          kk[j] = kj.x;
          kk[j + 1] = kj.y;
#pragma unroll
          for (int c = 0; c < C; ++c) {
            S[c][j] = mul2(S[c][j], gg.x);
            S[c][j + 1] = mul2(S[c][j + 1], gg.y);
            held[c][0] = fma2(S[c][j], kj.x, held[c][0]);
            held[c][1] = fma2(S[c][j + 1], kj.y, held[c][1]);
            acc[c][0] = fma2(S[c][j], qq.x, acc[c][0]);
            acc[c][1] = fma2(S[c][j + 1], qq.y, acc[c][1]);
          }
        }
        float h[C], u[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          h[c] = (low(held[c][0]) + high(held[c][0])) + (low(held[c][1]) + high(held[c][1]));
          o[c] = (low(acc[c][0]) + high(acc[c][0])) + (low(acc[c][1]) + high(acc[c][1]));
        }
#pragma unroll
        for (int x = LPC / 2; x > 0; x >>= 1)
#pragma unroll
          for (int c = 0; c < C; ++c) {
            h[c] += __shfl_xor_sync(~0u, h[c], x);
            o[c] += __shfl_xor_sync(~0u, o[c], x);
          }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          u[c] = __fmul_rn(beta, __fsub_rn(v[c], h[c]));
          o[c] = fmaf(u[c], kq, o[c]);  // S^T q behind the update: what the faded state held, and u (k . q)
          const pair uu = both(u[c]);
#pragma unroll
          for (int j = 0; j < P; ++j) S[c][j] = fma2(kk[j], uu, S[c][j]);
        }
      } else {
#pragma unroll
        for (int j = 0; j < P; j += 2) {
          const ulonglong2 kj = k4[LPC * (j / 2)], qq = q4[LPC * (j / 2)];
#pragma unroll
          for (int c = 0; c < C; ++c) {
            const pair kv = both(__fmul_rn(v[c], m.k_scale));
            S[c][j] = fma2(kj.x, kv, mul2(S[c][j], decay));
            S[c][j + 1] = fma2(kj.y, kv, mul2(S[c][j + 1], decay));
            acc[c][0] = fma2(S[c][j], qq.x, acc[c][0]);
            acc[c][1] = fma2(S[c][j + 1], qq.y, acc[c][1]);
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) o[c] = (low(acc[c][0]) + high(acc[c][0])) + (low(acc[c][1]) + high(acc[c][1]));
#pragma unroll
        for (int x = LPC / 2; x > 0; x >>= 1)
#pragma unroll
          for (int c = 0; c < C; ++c) o[c] += __shfl_xor_sync(~0u, o[c], x);
      }
      if (l == 0)
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (col + c < live) o_row[c] = o[c];
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
    if (col + c < live)
#pragma unroll
      for (int j = 0; j < P; j += 2) {
        const int i = 4 * (l + LPC * (j / 2));
        float* p = st + c * m.dim;
        const float4 v = make_float4(low(S[c][j]), high(S[c][j]), low(S[c][j + 1]), high(S[c][j + 1]));
        if (st_vec) {
          if (i < m.dim) *(float4*)(p + i) = v;
        } else {
          if (i < m.dim) p[i] = v.x;
          if (i + 1 < m.dim) p[i + 1] = v.y;
          if (i + 2 < m.dim) p[i + 2] = v.z;
          if (i + 3 < m.dim) p[i + 3] = v.w;
        }
      }
  if (whole) {  // the block holds the head: its norm and gate here
    __syncthreads();
    for (int r = tid >> 5; r < n; r += nt >> 5)
      head_out(o_raw + ((int64_t)(g.t0 + r) * m.n_head + head) * m.vdim, m.vdim, ho, g.t0 + r, head, tid & 31);
  }
}

// The scan over blocks of four rows: grid (column group, head, group of rows), cols / C * LPC threads, LPC lanes hold C columns.
// The 4 C dot products of a lane group end spread over its lanes: lane index -> (column, row of the block).
constexpr int BLOCK_STAGES = 4;
template <int DP, bool DELTA>
struct BlockLay {
  static constexpr int REC = rec_floats(DP, DELTA);
  static __host__ __device__ int stage(int cols) { return REC + BLOCK_ROWS * cols; }
  static __host__ __device__ int total(int cols, int lanes_all) { return BLOCK_STAGES * stage(cols) + 2 * lanes_all; }
};
template <int LPC, int R, int C, bool DELTA>
__global__ void __launch_bounds__(256)
block_scan_kernel(MatrixScan m, RowGroups groups, RowMap rows, int tokens, int cols, const float* __restrict__ rec, float* __restrict__ o_raw) {
  pdl_enter();
  constexpr int DP = LPC * R, P = R / 2, V = 4 * C, REP = LPC / V;
  static_assert(REP >= 1, "a lane per dot product");
  using L = BlockLay<DP, DELTA>;
  extern __shared__ __align__(16) float sm[];
  const Group g = group_of(groups, rows, tokens, blockIdx.z);
  const int tid = threadIdx.x, nt = blockDim.x, l = tid % LPC, grp = tid / LPC, col = grp * C, head = blockIdx.y;
  const int c0 = blockIdx.x * cols, live = min(cols, m.vdim - c0), stage = L::stage(cols);
  const int my_c = l / REP / 4, my_i = l / REP % 4;  // the product this lane ends up with
  float* xd = sm + BLOCK_STAGES * stage + grp * V;
  float* xu = xd + nt / LPC * V;
  const int n = g.t1 - g.t0, steps = (n + BLOCK_ROWS - 1) / BLOCK_ROWS;
  const float* src = rec + ((int64_t)first_block(groups, blockIdx.z) * m.n_head + head) * L::REC;
  const float* v_row = m.v + (int64_t)g.t0 * m.v_ld + (int64_t)head * m.vdim + c0;
  const bool v_vec = ((m.vdim | (int)m.v_ld | cols) & 3) == 0 && ((uintptr_t)m.v & 15) == 0;
  auto fetch = [&](int s) {
    float* base = sm + (s % BLOCK_STAGES) * stage;
    const float* from = src + (int64_t)s * m.n_head * L::REC;
    for (int i = 4 * tid; i < L::REC; i += 4 * nt) async16(base + i, from + i);
    float* sv = base + L::REC;
    const int nr = min(BLOCK_ROWS, n - s * BLOCK_ROWS);
    const float* vs = v_row + (int64_t)s * BLOCK_ROWS * m.v_ld;
    for (int i = tid; i < cols; i += nt) {  // a row of four values, or a column of the four rows
      if (v_vec) {
        const int r = i / (cols / 4), c = 4 * (i % (cols / 4));
        if (r < nr && c < live) async16(sv + r * cols + c, vs + r * m.v_ld + c);
        else *(float4*)(sv + r * cols + c) = make_float4(0.f, 0.f, 0.f, 0.f);
      } else {
        for (int r = 0; r < BLOCK_ROWS; ++r)
          if (r < nr && i < live) async4(sv + r * cols + i, vs + r * m.v_ld + i);
          else sv[r * cols + i] = 0.f;
      }
    }
    async_commit();
  };
#pragma unroll
  for (int s = 0; s < BLOCK_STAGES - 1; ++s) {
    if (s < steps) fetch(s);
    else async_commit();
  }
  float* st = m.state.state + g.seq * m.state.stride + ((int64_t)head * m.vdim + c0 + col) * m.dim;
  pair S[C][P];
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int j = 0; j < P; j += 2) {
      const int i = 4 * (l + LPC * (j / 2));
      ulonglong2 v = make_ulonglong2(0, 0);
      if (col + c < live && !g.fresh && i < m.dim) v = *(const ulonglong2*)(st + c * m.dim + i);
      S[c][j] = v.x;
      S[c][j + 1] = v.y;
    }
  if (DELTA) conv_tail_update(m.conv_in, m.conv_ld, m.conv, g, (blockIdx.y * gridDim.x + blockIdx.x) * nt + tid, (int)(gridDim.x * gridDim.y) * nt);
  // sums over the lanes of V values; the lane's own one is returned
  auto spread = [&](float (&val)[V]) {
    int w = V;
#pragma unroll
    for (int x = LPC / 2; x > 0; x >>= 1) {
      if (w > 1) {
        w /= 2;
        const bool up = l & x;
#pragma unroll
        for (int i = 0; i < V / 2; ++i)
          if (i < w) {
            const float keep = up ? val[i + w] : val[i], send = up ? val[i] : val[i + w];
            val[i] = keep + __shfl_xor_sync(~0u, send, x);
          }
      } else {
        val[0] += __shfl_xor_sync(~0u, val[0], x);
      }
    }
    return val[0];
  };
  float* o_row = o_raw + ((int64_t)(g.t0 + my_i) * m.n_head + head) * m.vdim + c0 + col + my_c;
  const int64_t o_ld = (int64_t)BLOCK_ROWS * m.n_head * m.vdim;
  const bool out_live = l % REP == 0 && col + my_c < live;
  for (int s = 0; s < steps; ++s, o_row += o_ld) {
    async_wait<BLOCK_STAGES - 2>();
    __syncthreads();  // block s has arrived for every thread, and everyone is done with block s - 1
    if (s + BLOCK_STAGES - 1 < steps) fetch(s + BLOCK_STAGES - 1);
    else async_commit();
    const float* base = sm + (s % BLOCK_STAGES) * stage;
    const float* sc = base + rec_vectors(DELTA) * DP;
    const float* sv = base + L::REC + col;
    const ulonglong2* vec = (const ulonglong2*)base + l;  // vector i, values 4 (l + LPC j): vec[i * DP / 4 + LPC j]
    const float4 srow = *(const float4*)(sc + 4 * my_i);
    float d[V], e[V];
    {
      pair ad[V], ae[V];
#pragma unroll
      for (int i = 0; i < V; ++i) ad[i] = ae[i] = 0;
#pragma unroll
      for (int j = 0; j < P; j += 2)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if constexpr (DELTA) {
            const ulonglong2 k = vec[i * (DP / 4) + LPC * (j / 2)];
#pragma unroll
            for (int c = 0; c < C; ++c) ad[4 * c + i] = fma2(S[c][j + 1], k.y, fma2(S[c][j], k.x, ad[4 * c + i]));
          }
          const ulonglong2 q = vec[((DELTA ? 4 : 0) + i) * (DP / 4) + LPC * (j / 2)];
#pragma unroll
          for (int c = 0; c < C; ++c) ae[4 * c + i] = fma2(S[c][j + 1], q.y, fma2(S[c][j], q.x, ae[4 * c + i]));
        }
#pragma unroll
      for (int i = 0; i < V; ++i) { d[i] = low(ad[i]) + high(ad[i]); e[i] = low(ae[i]) + high(ae[i]); }
    }
    float u[4];  // of this lane's column
    float4 uc[C];
    if constexpr (DELTA) {
      xd[l / REP] = spread(d);
      const float oe = spread(e);
      __syncwarp();
      const float4 dd = *(const float4*)(xd + 4 * my_c), beta = *(const float4*)(sc + 32);
      const float4 c2 = *(const float4*)(sc + 20), c3 = *(const float4*)(sc + 24), c4 = *(const float4*)(sc + 28);
      const float* vc = sv + my_c;
      u[0] = beta.x * (vc[0] - dd.x);
      u[1] = beta.y * (vc[cols] - dd.y - c2.x * u[0]);
      u[2] = beta.z * (vc[2 * cols] - dd.z - c3.x * u[0] - c3.y * u[1]);
      u[3] = beta.w * (vc[3 * cols] - dd.w - c4.x * u[0] - c4.y * u[1] - c4.z * u[2]);
      xu[l / REP] = my_i < 2 ? (my_i == 0 ? u[0] : u[1]) : (my_i == 2 ? u[2] : u[3]);
      __syncwarp();
#pragma unroll
      for (int c = 0; c < C; ++c) uc[c] = *(const float4*)(xu + 4 * c);
      e[0] = oe;
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) u[i] = sv[i * cols + my_c];
#pragma unroll
      for (int c = 0; c < C; ++c) uc[c] = make_float4(sv[c], sv[cols + c], sv[2 * cols + c], sv[3 * cols + c]);
    }
    // the state behind the block
    const pair fade4 = DELTA ? 0 : both(sc[36]);
#pragma unroll
    for (int j = 0; j < P; j += 2) {
      ulonglong2 f;
      if constexpr (DELTA) f = vec[12 * (DP / 4) + LPC * (j / 2)];
      else f = make_ulonglong2(fade4, fade4);
#pragma unroll
      for (int c = 0; c < C; ++c) { S[c][j] = mul2(S[c][j], f.x); S[c][j + 1] = mul2(S[c][j + 1], f.y); }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const ulonglong2 k = vec[((DELTA ? 8 : 4) + i) * (DP / 4) + LPC * (j / 2)];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const pair uu = both(i == 0 ? uc[c].x : i == 1 ? uc[c].y : i == 2 ? uc[c].z : uc[c].w);
          S[c][j] = fma2(k.x, uu, S[c][j]);
          S[c][j + 1] = fma2(k.y, uu, S[c][j + 1]);
        }
      }
    }
    if constexpr (!DELTA) e[0] = spread(e);
    const float o = fmaf(srow.x, u[0], fmaf(srow.y, u[1], fmaf(srow.z, u[2], fmaf(srow.w, u[3], e[0]))));
    if (out_live && s * BLOCK_ROWS + my_i < n) *o_row = o;
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
    if (col + c < live)
#pragma unroll
      for (int j = 0; j < P; j += 2) {
        const int i = 4 * (l + LPC * (j / 2));
        if (i < m.dim) *(ulonglong2*)(st + c * m.dim + i) = make_ulonglong2(S[c][j], S[c][j + 1]);
      }
}

// ---- gated linear recurrence per channel ------------------------------------------------------------------------------------
// grid (GS_COLS channels, group of rows).  GS_TILE rows at a time: all threads take the rows' decays and inputs, GS_COLS of them
// run along the rows, all write the results.
constexpr int GS_TILE = 128, GS_COLS = 16, GS_LANES = 16, GS_PER = GS_TILE / GS_LANES;  // GS_LANES threads per channel
__global__ void __launch_bounds__(GS_COLS * GS_LANES)
gated_scan_kernel(GatedScan p, RowGroups groups, RowMap rows, int tokens) {
  pdl_enter();
  __shared__ float2 ab[GS_TILE][GS_COLS];
  const Group g = group_of(groups, rows, tokens, blockIdx.y);
  const int lane = threadIdx.x % GS_COLS, first = threadIdx.x / GS_COLS, c = blockIdx.x * GS_COLS + lane;
  const bool live = c < p.width, runs = live && first == 0;
  conv_tail_update(p.conv_in, p.conv_ld, p.conv, g, blockIdx.x * blockDim.x + threadIdx.x, (int)(gridDim.x * blockDim.x));
  float* st = p.state.state + g.seq * p.state.stride + c;
  float S = runs && !g.fresh ? *st : 0.f;
  const int rg = live ? c / p.block * 2 * p.block + c % p.block : 0;  // the channel's r in a row of gates; i stands block further on
  const float rate = live ? p.rate[c] : 0.f, rb = live ? p.gate_bias[rg] : 0.f, ib = live ? p.gate_bias[rg + p.block] : 0.f, yb = live ? p.y_bias[c] : 0.f;
  for (int t0 = g.t0; t0 < g.t1; t0 += GS_TILE) {
    const int n = min(GS_TILE, g.t1 - t0);
    float gr[GS_PER], gi[GS_PER], u[GS_PER], y[GS_PER];
#pragma unroll
    for (int j = 0; j < GS_PER; ++j) {  // everything of the tile in flight at once
      const int r = first + j * GS_LANES;
      const int64_t t = t0 + r;
      const bool ok = live && r < n;
      gr[j] = ok ? p.gates[t * 2 * p.width + rg] : 0.f;
      gi[j] = ok ? p.gates[t * 2 * p.width + rg + p.block] : 0.f;
      u[j] = ok ? p.u[t * p.width + c] : 0.f;
      y[j] = ok ? p.y[t * p.y_ld + c] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < GS_PER; ++j) {
      const int r = first + j * GS_LANES;
      if (r >= n) break;
      const float log_a = -__fmul_rn(rate, sigmoid(__fadd_rn(gr[j], rb)));
      // a - 1 instead of a: a state that hardly fades would feel every rounding of a factor next to 1, at each of its steps
      const float less = expm1f(log_a), in = sqrtf(-__fmul_rn(less, 2.0f + less));  // 1 - a^2 = -(a - 1) (a + 1)
      ab[r][lane] = make_float2(less, __fmul_rn(__fmul_rn(in, sigmoid(__fadd_rn(gi[j], ib))), u[j]));
    }
    __syncthreads();
    if (runs) {
#pragma unroll 8
      for (int r = 0; r < n; ++r) {
        const float2 v = ab[r][lane];
        S = __fadd_rn(S, fmaf(v.x, S, v.y));
        ab[r][lane].x = S;
      }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < GS_PER; ++j) {
      const int r = first + j * GS_LANES;
      if (!live || r >= n) break;
      const int64_t t = t0 + r;
      const float v = __fmul_rn(__fmul_rn(ab[r][lane].x, gelu_tanh(__fadd_rn(y[j], yb))), p.scale);
      if (p.out) p.out[t * p.ld + c] = v;
      if (p.out16) ((__nv_bfloat16*)p.out16)[t * p.ld + c] = __float2bfloat16_rn(v);
    }
    __syncthreads();
  }
  if (runs) *st = S;
}

constexpr int SCAN_SHORT = 16, SCAN_BLOCKS = 120, BLOCK_GROUPS = 64;  // rows of a short group, blocks that fill the machine, most groups taken by blocks
bool by_blocks(int dim, const RowGroups& g) { return dim <= 128 && dim % 4 == 0 && g.longest > SCAN_SHORT && g.n <= BLOCK_GROUPS; }
int block_slots(int tokens, int groups) { return tokens / BLOCK_ROWS + groups; }
typedef void (*BlockKernel)(MatrixScan, RowGroups, RowMap, int, int, const float*, float*);
struct BlockChoice { BlockKernel kern; int lanes, per; };
template <int LPC, int R, int C>
BlockChoice block_choice(bool delta) { return BlockChoice{delta ? block_scan_kernel<LPC, R, C, true> : block_scan_kernel<LPC, R, C, false>, LPC, C}; }
// four columns per lane group where there are enough of them
BlockChoice block_of(int dim, bool delta, int64_t columns) {
  if (dim <= 32) return block_choice<8, 4, 2>(delta);
  if (dim <= 64) return columns >= 2400 ? block_choice<16, 4, 4>(delta) : block_choice<16, 4, 2>(delta);
  return columns >= 2400 ? block_choice<16, 8, 4>(delta) : block_choice<16, 8, 2>(delta);
}
int block_total(int dp, bool delta, int cols, int lanes_all) {
  return BLOCK_STAGES * (rec_floats(dp, delta) + BLOCK_ROWS * cols) + 2 * lanes_all;
}
typedef void (*ScanKernel)(MatrixScan, HeadOut, RowGroups, RowMap, int, int, bool, float*);
struct ScanChoice { ScanKernel kern; int lanes, per, threads; };  // lanes per column group, columns per group, most threads
template <int LPC, int R, int C>
ScanChoice scan_choice(bool delta, int cols, size_t* smem) {
  *smem = sizeof(float) * (delta ? ScanLay<LPC * R, true>::total(cols) : ScanLay<LPC * R, false>::total(cols));
  return ScanChoice{delta ? matrix_scan_kernel<LPC, R, C, true> : matrix_scan_kernel<LPC, R, C, false>, LPC, C, scan_threads(R)};
}
ScanChoice scan_of(int dim, bool delta, int cols, size_t* smem) {
  if (dim <= 32) return scan_choice<8, 4, 2>(delta, cols, smem);
  if (dim <= 64) return scan_choice<8, 8, 2>(delta, cols, smem);
  if (dim <= 128) return scan_choice<8, 16, 2>(delta, cols, smem);
  if (dim <= 256) return scan_choice<8, 32, 1>(delta, cols, smem);
  return scan_choice<32, 32, 1>(delta, cols, smem);
}

}  // namespace

bool matrix_scan_supported(int dim, int vdim) { return dim > 0 && dim <= 1024 && vdim > 0 && vdim <= 1024; }

int delta_prep_floats(const DeltaShape& d) {
  return (2 * d.n_kv * d.dim + d.n_head * d.vdim + d.n_head * d.dim + d.n_head + d.n_kv + 3) & ~3;
}
size_t scan_record_floats(int n_head, int dim, bool delta, int tokens, int n_seq) {
  if (dim > 128 || dim % 4 != 0) return 0;
  return (size_t)block_slots(tokens, std::min(n_seq, BLOCK_GROUPS)) * n_head * rec_floats(padded_dim(dim), delta);
}
bool scan_by_blocks(int dim, int vdim, const RowGroups& groups) { return vdim % 4 == 0 && by_blocks(dim, groups); }

cudaError_t launch_delta_prepare(const float* proj, int64_t ld, const float* a, const float* b, const DeltaShape& d, const ConvShape& conv, float* prep,
                                 float* records, const RowGroups& groups, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (!matrix_scan_supported(d.dim, d.vdim)) return cudaErrorInvalidValue;
  if (launches) ++*launches;
  if (records) {
    if (!scan_by_blocks(d.dim, d.vdim, groups) || ld % 4 != 0 || (((uintptr_t)proj | (uintptr_t)a) & 15) != 0) return cudaErrorInvalidValue;
    const int slots = block_slots(tokens, groups.n);
    return launch_walk(delta_blocks_kernel, dim3(slots, d.n_head), dim3(32 * BLOCK_ROWS), 0, s, proj, ld, a, b, d, conv, padded_dim(d.dim), records, prep, groups,
                       rows, tokens);
  }
  const int share = d.n_head / d.n_kv, values = 2 * d.dim + share * (d.dim + d.vdim);
  return launch_walk(delta_prepare_kernel, dim3(tokens, d.n_kv), dim3(std::min(1024, (values + 31) / 32 * 32)), (size_t)2 * d.dim * sizeof(float), s, proj, ld, a,
                     b, d, conv, prep, (int64_t)delta_prep_floats(d), rows);
}

cudaError_t launch_conv_rows(const float* x, int64_t ld, const ConvShape& conv, float* u, void* u16, int block, const RowMap& rows, int tokens,
                             cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  const bool vec = ((conv.channels | block | (int)ld) & 3) == 0 &&
                   (((uintptr_t)x | (uintptr_t)u | (uintptr_t)conv.bias | (uintptr_t)conv.tail.state) & 15) == 0 && conv.tail.stride % 4 == 0;
  const int per = CONV_THREADS * (vec ? 4 : 1);
  return launch_walk(conv_rows_kernel, dim3(tokens, (conv.channels + per - 1) / per), dim3(CONV_THREADS), 0, s, x, ld, conv, u, (__nv_bfloat16*)u16, block, rows,
                     vec);
}

cudaError_t launch_triple_columns(const void* w, int64_t rows, int cols, void* out, cudaStream_t s, uint64_t* launches) {
  if (launches) ++*launches;
  triple_columns_kernel<<<(unsigned)std::min<int64_t>((rows * cols + 255) / 256, 1024), 256, 0, s>>>((const uint16_t*)w, rows * cols, cols, (uint16_t*)out);
  return cudaGetLastError();
}

static cudaError_t launch_block_scan(const MatrixScan& m, const HeadOut& out, float* records, const RowGroups& groups, const RowMap& rows, int tokens,
                                     float* o_scratch, cudaStream_t s, uint64_t* launches) {
  const bool delta = m.conv_in != nullptr;
  const int slots = block_slots(tokens, groups.n), dp = padded_dim(m.dim);
  if (!scan_by_blocks(m.dim, m.vdim, groups) || ((uintptr_t)m.state.state & 15) != 0 || m.state.stride % 4 != 0 || ((uintptr_t)records & 15) != 0)
    return cudaErrorInvalidValue;
  cudaError_t e;
  if (!delta) {
    if (m.ld % 4 != 0 || (((uintptr_t)m.q | (uintptr_t)m.k) & 15) != 0) return cudaErrorInvalidValue;
    if (launches) ++*launches;
    e = launch_walk(retention_blocks_kernel, dim3((unsigned)(((int64_t)slots * m.n_head + 3) / 4)), dim3(128), 0, s, m, dp, records, groups, tokens, slots);
    if (e != cudaSuccess) return e;
  }
  const BlockChoice c = block_of(m.dim, delta, (int64_t)m.n_head * m.vdim * groups.n);
  const int warp_cols = 32 / c.lanes * c.per, most = 256 / c.lanes * c.per, whole = (m.vdim + warp_cols - 1) / warp_cols * warp_cols;
  int cols = std::min(whole, most);
  while (cols > warp_cols && (int64_t)m.n_head * groups.n * ((m.vdim + cols - 1) / cols) < SCAN_BLOCKS) cols = (cols / warp_cols + 1) / 2 * warp_cols;
  const int threads = cols / c.per * c.lanes;
  const size_t smem = (size_t)block_total(dp, delta, cols, threads) * sizeof(float);
  if (smem > 48 * 1024) {
    e = cudaFuncSetAttribute((const void*)c.kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  if (launches) *launches += 2;
  // Not placed while its predecessor runs, unlike the walk's other kernels: one block per SM for long is the whole plan, and blocks
  // that start early crowd onto the SMs that happen to be free.
  c.kern<<<dim3((m.vdim + cols - 1) / cols, m.n_head, groups.n), threads, smem, s>>>(m, groups, rows, tokens, cols, records, o_scratch);
  if ((e = cudaGetLastError()) != cudaSuccess) return e;
  return launch_walk(head_out_kernel, dim3((unsigned)(((int64_t)tokens * m.n_head + 7) / 8)), dim3(256), 0, s, (const float*)o_scratch, m.n_head, m.vdim, out,
                     tokens);
}

cudaError_t launch_matrix_scan(const MatrixScan& m, const HeadOut& out, float* records, const RowGroups& groups, const RowMap& rows, int tokens,
                               float* o_scratch, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (!matrix_scan_supported(m.dim, m.vdim) || m.n_head % m.n_kv != 0 || (m.rot.dims > 0 && tokens != 1)) return cudaErrorInvalidValue;
  if (records) return launch_block_scan(m, out, records, groups, rows, tokens, o_scratch, s, launches);
  const bool delta = m.g != nullptr;
  size_t smem = 0;
  const ScanChoice c = scan_of(m.dim, delta, 0, &smem);
  // Whole heads per block for short groups (norm and gate in the same launch); for long ones columns spread over the SMs, as
  // many per block as still fill them, since every block of a head stages its queries and keys.  Columns come as whole warps.
  const int warp_cols = 32 / c.lanes * c.per, most = c.threads / c.lanes * c.per, whole = (m.vdim + warp_cols - 1) / warp_cols * warp_cols;
  int cols = std::min(whole, most / warp_cols * warp_cols);
  if (groups.longest > SCAN_SHORT)
    while (cols > warp_cols && (int64_t)m.n_head * groups.n * ((m.vdim + cols - 1) / cols) < SCAN_BLOCKS) cols = (cols / warp_cols + 1) / 2 * warp_cols;
  scan_of(m.dim, delta, cols, &smem);
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute((const void*)c.kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  const int parts = (m.vdim + cols - 1) / cols;
  const bool fused = parts == 1 && groups.longest <= SCAN_SHORT;
  if (launches) *launches += fused ? 1 : 2;
  cudaError_t e = launch_walk(c.kern, dim3(parts, m.n_head, groups.n), dim3(cols / c.per * c.lanes), smem, s, m, out, groups, rows, tokens, cols, fused, o_scratch);
  if (e != cudaSuccess || fused) return e;
  const int64_t heads = (int64_t)tokens * m.n_head;
  return launch_walk(head_out_kernel, dim3((unsigned)((heads + 7) / 8)), dim3(256), 0, s, (const float*)o_scratch, m.n_head, m.vdim, out, tokens);
}

cudaError_t launch_gated_scan(const GatedScan& g, const RowGroups& groups, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  const dim3 grid((g.width + GS_COLS - 1) / GS_COLS, groups.n);
  if (groups.longest <= SCAN_SHORT) return launch_walk(gated_scan_kernel, grid, dim3(GS_COLS * GS_LANES), 0, s, g, groups, rows, tokens);
  gated_scan_kernel<<<grid, GS_COLS * GS_LANES, 0, s>>>(g, groups, rows, tokens);  // not placed early, as above
  return cudaGetLastError();
}

}  // namespace llr
