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

__device__ __forceinline__ float sigmoid(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }
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
// channel c at row t; near: rows_before(t, taps - 1), pos: the row's position
__device__ __forceinline__ float conv_at(const float* x, int64_t ld, const ConvShape& cv, const float* tail, int t, int near, int pos, int c) {
  const float* w = cv.w + (int64_t)c * cv.taps;
  const float b = cv.bias ? cv.bias[c] : 0.f;
  float acc = 0.f;
  for (int j = cv.taps - 1; j >= 0; --j) {  // oldest input first
    float v = 0.f;
    if (j <= near) v = __fadd_rn(x[(int64_t)(t - j) * ld + c], b);
    else if (j <= pos) v = tail[(int64_t)(cv.taps - 1 - (j - near)) * cv.channels + c];
    acc = fmaf(w[cv.taps - 1 - j], v, acc);
  }
  return cv.out_bias ? __fadd_rn(acc, cv.out_bias[c]) : acc;
}
// The last taps - 1 inputs behind the group's rows become the state's; thread `at` of `all` owns every all-th channel.
__device__ __forceinline__ void conv_tail_update(const float* x, int64_t ld, const ConvShape& cv, const Group& g, int at, int all) {
  if (cv.taps < 2) return;
  float* tail = cv.tail.state + g.seq * cv.tail.stride;
  const int keep = cv.taps - 1, n = g.t1 - g.t0;
  for (int c = at; c < cv.channels; c += all) {
    const float b = cv.bias ? cv.bias[c] : 0.f;
    for (int k = 0; k < keep; ++k) {  // ascending: what moves down is read before it is written
      const int back = keep - k;      // rows before the next one
      float v;
      if (back <= n) v = __fadd_rn(x[(int64_t)(g.t1 - back) * ld + c], b);
      else v = g.fresh ? 0.f : tail[(int64_t)(k + n) * cv.channels + c];
      tail[(int64_t)k * cv.channels + c] = v;
    }
  }
}

// one block per row and CONV_COLS channels
constexpr int CONV_COLS = 1024;
__global__ void __launch_bounds__(256)
conv_rows_kernel(const float* __restrict__ x, int64_t ld, ConvShape cv, float* __restrict__ u, __nv_bfloat16* __restrict__ u16, int block, RowMap rows) {
  pdl_enter();
  const int t = blockIdx.x, near = rows_before(rows, t, cv.taps - 1), pos = row_position(rows, t);
  const float* tail = cv.tail.state + row_sequence(rows, t) * cv.tail.stride;
  const int c1 = min(cv.channels, (int)(blockIdx.y + 1) * CONV_COLS);
  for (int c = blockIdx.y * CONV_COLS + threadIdx.x; c < c1; c += 256) {
    const float v = conv_at(x, ld, cv, tail, t, near, pos, c);
    u[(int64_t)t * cv.channels + c] = v;
    if (u16) {  // v as a sum of three bfloat16 values: 24 bits of mantissa
      __nv_bfloat16* o = u16 + (int64_t)t * 3 * cv.channels + (int64_t)(c / block) * 3 * block + c % block;
      const __nv_bfloat16 hi = __float2bfloat16_rn(v);
      const float r1 = __fsub_rn(v, __bfloat162float(hi));
      const __nv_bfloat16 mid = __float2bfloat16_rn(r1);
      o[0] = hi;
      o[block] = mid;
      o[2 * block] = __float2bfloat16_rn(__fsub_rn(r1, __bfloat162float(mid)));
    }
  }
}

__global__ void triple_columns_kernel(const uint16_t* __restrict__ w, int64_t n, int cols, uint16_t* __restrict__ out) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t at = i / cols * 3 * cols + i % cols;
    out[at] = out[at + cols] = out[at + 2 * cols] = w[i];
  }
}

// ---- inputs of the delta rule -------------------------------------------------------------------------------------------
// one block per row
constexpr int PREP_THREADS = 512;
__global__ void __launch_bounds__(PREP_THREADS)
delta_prepare_kernel(const float* __restrict__ proj, int64_t ld, const float* __restrict__ a, const float* __restrict__ b, DeltaShape d, ConvShape cv,
                     float* __restrict__ prep, int64_t prep_ld, RowMap rows) {
  pdl_enter();
  extern __shared__ float qk[];  // q | k of the row behind convolution and silu
  const int t = blockIdx.x, near = rows_before(rows, t, cv.taps - 1), pos = row_position(rows, t);
  const float* tail = cv.tail.state + row_sequence(rows, t) * cv.tail.stride;
  const int nq = d.n_kv * d.dim, nv = d.n_head * d.vdim, ng = d.n_head * d.dim;
  float* o = prep + (int64_t)t * prep_ld;
  for (int c = threadIdx.x; c < 2 * nq + nv; c += PREP_THREADS) {
    const float z = conv_at(proj, ld, cv, tail, t, near, pos, c), v = __fdiv_rn(z, 1.0f + expf(-z));
    if (c < 2 * nq) qk[c] = v;
    else o[c] = v;
  }
  for (int c = threadIdx.x; c < ng; c += PREP_THREADS)
    o[2 * nq + nv + c] = expf(-__fmul_rn(d.rate[c / d.dim], softplus(__fadd_rn(a[(int64_t)t * ng + c], d.step_bias[c]))));
  for (int h = threadIdx.x; h < d.n_head; h += PREP_THREADS) o[2 * nq + nv + ng + h] = sigmoid(b[(int64_t)t * ld + h]);
  __syncthreads();
  const int lane = threadIdx.x & 31;
  for (int g = threadIdx.x >> 5; g < d.n_kv; g += PREP_THREADS / 32) {  // a warp per head
    const float *q = qk + g * d.dim, *k = qk + nq + g * d.dim;
    float sq = 0.f, sk = 0.f;
    for (int i = lane; i < d.dim; i += 32) { sq = fmaf(q[i], q[i], sq); sk = fmaf(k[i], k[i], sk); }
    sq = sqrtf(__fadd_rn(warp_sum(sq), d.unit_eps));
    sk = sqrtf(__fadd_rn(warp_sum(sk), d.unit_eps));
    float kq = 0.f;
    for (int i = lane; i < d.dim; i += 32) {
      const float qv = __fmul_rn(__fdiv_rn(q[i], sq), d.q_scale), kv = __fdiv_rn(k[i], sk);
      o[g * d.dim + i] = qv;
      o[nq + g * d.dim + i] = kv;
      kq = fmaf(kv, qv, kq);
    }
    kq = warp_sum(kq);
    if (lane == 0) o[2 * nq + nv + ng + d.n_head + g] = kq;
  }
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

// a head's result behind its norm and gate; a warp per head and row.  o: vdim values in shared or global memory
__device__ __forceinline__ void head_out(const float* o, int vdim, const HeadOut& ho, int t, int h, int lane) {
  float ss = 0.f;
  for (int i = lane; i < vdim; i += 32) ss = fmaf(o[i], o[i], ss);
  const float rms = sqrtf(__fadd_rn(__fdiv_rn(warp_sum(ss), (float)vdim), ho.eps));
  for (int i = lane; i < vdim; i += 32) {
    float v = __fdiv_rn(o[i], rms);
    if (ho.weight) v = __fmul_rn(v, ho.weight[i]);
    const float g = ho.gate[(int64_t)t * ho.gate_ld + (int64_t)h * vdim + i];
    v = __fmul_rn(__fmul_rn(v, ho.silu ? __fmul_rn(g, sigmoid(g)) : sigmoid(g)), ho.scale);
    const int64_t at = (int64_t)t * ho.ld + (int64_t)h * vdim + i;
    if (ho.out) ho.out[at] = v;
    if (ho.out16) ((__nv_bfloat16*)ho.out16)[at] = __float2bfloat16_rn(v);
  }
}
__global__ void __launch_bounds__(256)
head_out_kernel(const float* __restrict__ o, int heads, int vdim, HeadOut ho, int tokens) {
  pdl_enter();
  const int64_t i = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= (int64_t)tokens * heads) return;
  head_out(o + i * vdim, vdim, ho, (int)(i / heads), (int)(i % heads), threadIdx.x & 31);
}

constexpr int SCAN_STAGES = 3;  // stages in flight
// Shared memory of a block, in floats: per stage q | k (| g) of DP values per row, v and one pair (beta, k . q) per row; then
// the stage's results where the block holds whole heads
template <int DP, bool DELTA>
struct ScanLay {
  static constexpr int VEC = DP * (DELTA ? 3 : 2), ROWS = DP > 256 ? 2 : 8;  // rows per stage
  static __host__ __device__ int stage(int cols) { return ROWS * (VEC + ((cols + 3) & ~3) + 4); }
  static __host__ __device__ int total(int cols) { return SCAN_STAGES * stage(cols) + ROWS * cols; }
};
constexpr int scan_threads(int lpc, int r) { return lpc * r > 128 ? 512 : 1024; }  // most threads of a block: the state stays in registers

// grid (column group, head, group of rows); cols * LPC threads.  LPC lanes hold a column: lane l the values 4 (l + LPC j) + c.
template <int LPC, int R, bool DELTA>
__global__ void __launch_bounds__(scan_threads(LPC, R))
matrix_scan_kernel(MatrixScan m, HeadOut ho, RowGroups groups, RowMap rows, int tokens, int cols, float* __restrict__ o_raw) {
  pdl_enter();
  constexpr int DP = LPC * R;
  using L = ScanLay<DP, DELTA>;
  constexpr int SCAN_ROWS = L::ROWS;
  extern __shared__ __align__(16) float sm[];
  const Group g = group_of(groups, rows, tokens, blockIdx.z);
  const int tid = threadIdx.x, nt = blockDim.x, l = tid % LPC, col = tid / LPC, head = blockIdx.y, kvh = head / (m.n_head / m.n_kv);
  const int c0 = blockIdx.x * cols, live = min(cols, m.vdim - c0), stage = L::stage(cols), v_ld = (cols + 3) & ~3;
  const bool fused = gridDim.x == 1;
  float* so = sm + SCAN_STAGES * stage;
  if (DELTA) conv_tail_update(m.conv_in, m.conv_ld, m.conv, g, (blockIdx.y * gridDim.x + blockIdx.x) * nt + tid, (int)(gridDim.x * gridDim.y) * nt);
  // values behind dim stay zero
  if (m.dim < DP)
    for (int i = tid; i < SCAN_STAGES * stage; i += nt) sm[i] = 0.f;
  const bool vec = ((m.dim | (int)m.ld) & 3) == 0 && (((uintptr_t)m.q | (uintptr_t)m.k | (DELTA ? (uintptr_t)m.g : 0)) & 15) == 0;
  if (m.dim < DP) __syncthreads();
  const int n = g.t1 - g.t0, steps = (n + SCAN_ROWS - 1) / SCAN_ROWS;
  auto fetch = [&](int s) {
    float* base = sm + (s % SCAN_STAGES) * stage;
    const int r0 = g.t0 + s * SCAN_ROWS, nr = min(SCAN_ROWS, g.t1 - r0);
    auto run = [&](float* dst, const float* src, int64_t ld) {  // nr rows of dim values, DP apart
      if (vec) {
        const int w = m.dim / 4;
        for (int i = tid; i < nr * w; i += nt) async16(dst + i / w * DP + 4 * (i % w), src + (i / w) * ld + 4 * (i % w));
      } else {
        for (int i = tid; i < nr * m.dim; i += nt) async4(dst + i / m.dim * DP + i % m.dim, src + (i / m.dim) * ld + i % m.dim);
      }
    };
    if (m.rot.dims > 0) {  // a single row as the product left it
      const int half = m.rot.dims / 2;
      for (int i = tid; i < 2 * m.dim; i += nt) {
        const bool key = i >= m.dim;
        const int c = key ? i - m.dim : i;
        const float* src = (key ? m.k : m.q) + (int64_t)r0 * m.ld + (int64_t)kvh * m.dim;
        float v = src[c];
        if (c < 2 * half) {
          const float2 a = m.rot.cs[(int64_t)r0 * m.rot.ld + (c < half ? c : c - half)];
          v = c < half ? fmaf(v, a.x, -__fmul_rn(src[c + half], a.y)) : fmaf(v, a.x, __fmul_rn(src[c - half], a.y));
        }
        base[(key ? SCAN_ROWS * DP : 0) + c] = v;
      }
    } else {
      run(base, m.q + (int64_t)r0 * m.ld + (int64_t)kvh * m.dim, m.ld);
      run(base + SCAN_ROWS * DP, m.k + (int64_t)r0 * m.ld + (int64_t)kvh * m.dim, m.ld);
    }
    if (DELTA) run(base + 2 * SCAN_ROWS * DP, m.g + (int64_t)r0 * m.ld + (int64_t)head * m.dim, m.ld);
    float* sv = base + SCAN_ROWS * L::VEC;
    for (int i = tid; i < nr * live; i += nt) async4(sv + i / live * v_ld + i % live, m.v + (int64_t)(r0 + i / live) * m.v_ld + (int64_t)head * m.vdim + c0 + i % live);
    if (DELTA && tid < nr) {
      async4(sv + SCAN_ROWS * v_ld + 2 * tid, m.beta + (int64_t)(r0 + tid) * m.ld + head);
      async4(sv + SCAN_ROWS * v_ld + 2 * tid + 1, m.kq + (int64_t)(r0 + tid) * m.ld + kvh);
    }
    async_commit();
  };
#pragma unroll
  for (int s = 0; s < SCAN_STAGES - 1; ++s) {
    if (s < steps) fetch(s);
    else async_commit();
  }
  // the column's state
  float* st = m.state.state + g.seq * m.state.stride + ((int64_t)head * m.vdim + c0 + col) * m.dim;
  const bool mine = col < live, st_vec = (m.dim & 3) == 0 && ((uintptr_t)st & 15) == 0;
  float4 S[R / 4];
#pragma unroll
  for (int j = 0; j < R / 4; ++j) {
    const int i = 4 * (l + LPC * j);
    S[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (mine && !g.fresh) {
      if (st_vec) {
        if (i < m.dim) S[j] = *(const float4*)(st + i);
      } else {
        if (i < m.dim) S[j].x = st[i];
        if (i + 1 < m.dim) S[j].y = st[i + 1];
        if (i + 2 < m.dim) S[j].z = st[i + 2];
        if (i + 3 < m.dim) S[j].w = st[i + 3];
      }
    }
  }
  const float decay = DELTA ? 0.f : m.decay[head];
  for (int s = 0; s < steps; ++s) {
    async_wait<SCAN_STAGES - 2>();
    __syncthreads();  // stage s has arrived for every thread, and everyone is done with stage s - 1
    if (s + SCAN_STAGES - 1 < steps) fetch(s + SCAN_STAGES - 1);
    else async_commit();
    const float* base = sm + (s % SCAN_STAGES) * stage;
    const float* sv = base + SCAN_ROWS * L::VEC;
    const int r0 = g.t0 + s * SCAN_ROWS, nr = min(SCAN_ROWS, g.t1 - r0);
#pragma unroll (R <= 8 ? 2 : 1)
    for (int r = 0; r < nr; ++r) {
      const float4* q4 = (const float4*)(base + r * DP) + l;
      const float4* k4 = (const float4*)(base + (SCAN_ROWS + r) * DP) + l;
      const float v = sv[r * v_ld + min(col, cols - 1)];
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      float o;
      if constexpr (DELTA) {
        const float4* g4 = (const float4*)(base + (2 * SCAN_ROWS + r) * DP) + l;
        const float beta = sv[SCAN_ROWS * v_ld + 2 * r], kq = sv[SCAN_ROWS * v_ld + 2 * r + 1];
        float4 held = make_float4(0.f, 0.f, 0.f, 0.f);
        float4 kk[R / 4];
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
          const float4 gg = g4[LPC * j], qq = q4[LPC * j];
          kk[j] = k4[LPC * j];
          S[j].x = __fmul_rn(S[j].x, gg.x); S[j].y = __fmul_rn(S[j].y, gg.y); S[j].z = __fmul_rn(S[j].z, gg.z); S[j].w = __fmul_rn(S[j].w, gg.w);
          held.x = fmaf(S[j].x, kk[j].x, held.x); held.y = fmaf(S[j].y, kk[j].y, held.y);
          held.z = fmaf(S[j].z, kk[j].z, held.z); held.w = fmaf(S[j].w, kk[j].w, held.w);
          acc.x = fmaf(S[j].x, qq.x, acc.x); acc.y = fmaf(S[j].y, qq.y, acc.y);
          acc.z = fmaf(S[j].z, qq.z, acc.z); acc.w = fmaf(S[j].w, qq.w, acc.w);
        }
        float hs = (held.x + held.y) + (held.z + held.w);
        o = (acc.x + acc.y) + (acc.z + acc.w);
#pragma unroll
        for (int x = LPC / 2; x > 0; x >>= 1) hs += __shfl_xor_sync(~0u, hs, x);
        const float u = __fmul_rn(beta, __fsub_rn(v, hs));
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
          S[j].x = fmaf(kk[j].x, u, S[j].x); S[j].y = fmaf(kk[j].y, u, S[j].y); S[j].z = fmaf(kk[j].z, u, S[j].z); S[j].w = fmaf(kk[j].w, u, S[j].w);
        }
#pragma unroll
        for (int x = LPC / 2; x > 0; x >>= 1) o += __shfl_xor_sync(~0u, o, x);
        o = fmaf(u, kq, o);  // S^T q behind the update: what the faded state held, and u (k . q)
      } else {
        const float kv = __fmul_rn(v, m.k_scale);
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
          const float4 kj = k4[LPC * j], qq = q4[LPC * j];
          S[j].x = fmaf(kj.x, kv, __fmul_rn(S[j].x, decay)); S[j].y = fmaf(kj.y, kv, __fmul_rn(S[j].y, decay));
          S[j].z = fmaf(kj.z, kv, __fmul_rn(S[j].z, decay)); S[j].w = fmaf(kj.w, kv, __fmul_rn(S[j].w, decay));
          acc.x = fmaf(S[j].x, qq.x, acc.x); acc.y = fmaf(S[j].y, qq.y, acc.y);
          acc.z = fmaf(S[j].z, qq.z, acc.z); acc.w = fmaf(S[j].w, qq.w, acc.w);
        }
        o = (acc.x + acc.y) + (acc.z + acc.w);
#pragma unroll
        for (int x = LPC / 2; x > 0; x >>= 1) o += __shfl_xor_sync(~0u, o, x);
      }
      if (l == 0 && mine) {
        if (fused) so[r * cols + col] = o;
        else o_raw[((int64_t)(r0 + r) * m.n_head + head) * m.vdim + c0 + col] = o;
      }
    }
    if (fused) {
      __syncthreads();
      if ((nt & 31) == 0)
        for (int r = tid >> 5; r < nr; r += nt >> 5) head_out(so + r * cols, m.vdim, ho, r0 + r, head, tid & 31);
    }
  }
  if (mine) {
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
      const int i = 4 * (l + LPC * j);
      if (st_vec) {
        if (i < m.dim) *(float4*)(st + i) = S[j];
      } else {
        if (i < m.dim) st[i] = S[j].x;
        if (i + 1 < m.dim) st[i + 1] = S[j].y;
        if (i + 2 < m.dim) st[i + 2] = S[j].z;
        if (i + 3 < m.dim) st[i + 3] = S[j].w;
      }
    }
  }
}

// ---- gated linear recurrence per channel ------------------------------------------------------------------------------------
// grid (32 channels, group of rows).  TILE rows at a time: the warps take the rows' decays and inputs, one warp runs along
// them, the warps write the results.
constexpr int GS_TILE = 128, GS_WARPS = 16;
__global__ void __launch_bounds__(32 * GS_WARPS)
gated_scan_kernel(GatedScan p, RowGroups groups, RowMap rows, int tokens) {
  pdl_enter();
  __shared__ float2 ab[GS_TILE][32];
  const Group g = group_of(groups, rows, tokens, blockIdx.y);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
  const bool live = c < p.width;
  conv_tail_update(p.conv_in, p.conv_ld, p.conv, g, blockIdx.x * blockDim.x + threadIdx.x, (int)(gridDim.x * blockDim.x));
  float* st = p.state.state + g.seq * p.state.stride + c;
  float S = live && !g.fresh && warp == 0 ? *st : 0.f;
  const int rg = live ? c / p.block * 2 * p.block + c % p.block : 0;  // the channel's r in a row of gates; i stands block further on
  const float rate = live ? p.rate[c] : 0.f, rb = live ? p.gate_bias[rg] : 0.f, ib = live ? p.gate_bias[rg + p.block] : 0.f, yb = live ? p.y_bias[c] : 0.f;
  for (int t0 = g.t0; t0 < g.t1; t0 += GS_TILE) {
    const int n = min(GS_TILE, g.t1 - t0);
    if (live) {
#pragma unroll 4
      for (int r = warp; r < n; r += GS_WARPS) {
        const int64_t t = t0 + r;
        const float* gr = p.gates + t * 2 * p.width + rg;
        const float log_a = -__fmul_rn(rate, sigmoid(__fadd_rn(gr[0], rb)));
        // 1 - a^2 without the cancellation near a = 1
        const float in = sqrtf(-expm1f(2.0f * log_a));
        ab[r][lane] = make_float2(expf(log_a), __fmul_rn(__fmul_rn(in, sigmoid(__fadd_rn(gr[p.block], ib))), p.u[t * p.width + c]));
      }
    }
    __syncthreads();
    if (warp == 0) {
#pragma unroll 8
      for (int r = 0; r < n; ++r) {
        const float2 v = ab[r][lane];
        S = fmaf(v.x, S, v.y);
        ab[r][lane].x = S;
      }
    }
    __syncthreads();
    if (live) {
#pragma unroll 4
      for (int r = warp; r < n; r += GS_WARPS) {
        const int64_t t = t0 + r;
        const float v = __fmul_rn(__fmul_rn(ab[r][lane].x, gelu_tanh(__fadd_rn(p.y[t * p.y_ld + c], yb))), p.scale);
        if (p.out) p.out[t * p.ld + c] = v;
        if (p.out16) ((__nv_bfloat16*)p.out16)[t * p.ld + c] = __float2bfloat16_rn(v);
      }
    }
    __syncthreads();
  }
  if (live && warp == 0) *st = S;
}

constexpr int SCAN_SHORT = 16, SCAN_COLS = 16;  // rows of a short group, columns of a block for long ones
typedef void (*ScanKernel)(MatrixScan, HeadOut, RowGroups, RowMap, int, int, float*);
struct ScanChoice { ScanKernel kern; int lanes, floats, threads; };
template <int LPC, int R>
ScanChoice scan_choice(bool delta, int cols) {
  return delta ? ScanChoice{matrix_scan_kernel<LPC, R, true>, LPC, ScanLay<LPC * R, true>::total(cols), scan_threads(LPC, R)}
               : ScanChoice{matrix_scan_kernel<LPC, R, false>, LPC, ScanLay<LPC * R, false>::total(cols), scan_threads(LPC, R)};
}
ScanChoice scan_of(int dim, bool delta, int cols) {
  if (dim <= 32) return scan_choice<8, 4>(delta, cols);
  if (dim <= 64) return scan_choice<8, 8>(delta, cols);
  if (dim <= 128) return scan_choice<8, 16>(delta, cols);
  if (dim <= 256) return scan_choice<8, 32>(delta, cols);
  return scan_choice<32, 32>(delta, cols);
}

}  // namespace

bool matrix_scan_supported(int dim, int vdim) { return dim > 0 && dim <= 1024 && vdim > 0 && vdim <= 1024; }

int delta_prep_floats(const DeltaShape& d) {
  return (2 * d.n_kv * d.dim + d.n_head * d.vdim + d.n_head * d.dim + d.n_head + d.n_kv + 3) & ~3;
}
bool delta_supported(const DeltaShape& d) { return matrix_scan_supported(d.dim, d.vdim) && (size_t)2 * d.n_kv * d.dim * sizeof(float) <= 160 * 1024; }

cudaError_t launch_delta_prepare(const float* proj, int64_t ld, const float* a, const float* b, const DeltaShape& d, const ConvShape& conv, float* prep,
                                 const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (!delta_supported(d)) return cudaErrorInvalidValue;
  const size_t smem = (size_t)2 * d.n_kv * d.dim * sizeof(float);
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  if (launches) ++*launches;
  return launch_walk(delta_prepare_kernel, dim3(tokens), dim3(PREP_THREADS), smem, s, proj, ld, a, b, d, conv, prep, (int64_t)delta_prep_floats(d), rows);
}

cudaError_t launch_conv_rows(const float* x, int64_t ld, const ConvShape& conv, float* u, void* u16, int block, const RowMap& rows, int tokens,
                             cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(conv_rows_kernel, dim3(tokens, (conv.channels + CONV_COLS - 1) / CONV_COLS), dim3(256), 0, s, x, ld, conv, u, (__nv_bfloat16*)u16, block,
                     rows);
}

cudaError_t launch_triple_columns(const void* w, int64_t rows, int cols, void* out, cudaStream_t s, uint64_t* launches) {
  if (launches) ++*launches;
  triple_columns_kernel<<<(unsigned)std::min<int64_t>((rows * cols + 255) / 256, 1024), 256, 0, s>>>((const uint16_t*)w, rows * cols, cols, (uint16_t*)out);
  return cudaGetLastError();
}

cudaError_t launch_matrix_scan(const MatrixScan& m, const HeadOut& out, const RowGroups& groups, const RowMap& rows, int tokens, float* o_scratch,
                               cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (!matrix_scan_supported(m.dim, m.vdim) || m.n_head % m.n_kv != 0 || (m.rot.dims > 0 && tokens != 1)) return cudaErrorInvalidValue;
  const bool delta = m.g != nullptr;
  const ScanChoice any = scan_of(m.dim, delta, 1);
  const int lanes = any.lanes, warp_cols = 32 / lanes, most = any.threads / lanes;
  // Whole heads per block for short groups (norm and gate in the same launch) or short value rows; columns spread over the SMs
  // for long ones.  Columns of a block come as whole warps.
  const int whole = (m.vdim + warp_cols - 1) / warp_cols * warp_cols;
  const int cols = whole > most || (groups.longest > SCAN_SHORT && whole > SCAN_COLS) ? SCAN_COLS : whole;
  const ScanChoice c = scan_of(m.dim, delta, cols);
  const size_t smem = (size_t)c.floats * sizeof(float);
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute((const void*)c.kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  const int parts = (m.vdim + cols - 1) / cols;
  if (launches) *launches += parts > 1 ? 2 : 1;
  cudaError_t e = launch_walk(c.kern, dim3(parts, m.n_head, groups.n), dim3(cols * lanes), smem, s, m, out, groups, rows, tokens, cols, o_scratch);
  if (e != cudaSuccess || parts == 1) return e;
  const int64_t heads = (int64_t)tokens * m.n_head;
  return launch_walk(head_out_kernel, dim3((unsigned)((heads + 7) / 8)), dim3(256), 0, s, (const float*)o_scratch, m.n_head, m.vdim, out, tokens);
}

cudaError_t launch_gated_scan(const GatedScan& g, const RowGroups& groups, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches) {
  if (tokens <= 0) return cudaSuccess;
  if (launches) ++*launches;
  return launch_walk(gated_scan_kernel, dim3((g.width + 31) / 32, groups.n), dim3(32 * GS_WARPS), 0, s, g, groups, rows, tokens);
}

}  // namespace llr
