// Device helpers the kernels of the walks share (llr_decode.cu: the Llama walk; llr_mixers.cu: decoders described layer by
// layer): block sums, where a row of a batch stands, programmatic launches, and the attention of one row over one slice
// of keys.
#pragma once
#include <cuda_runtime.h>
#include <math_constants.h>

#include <cstdlib>

#include "llr_kernels.cuh"

namespace llr {
namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(~0u, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(~0u, v, o));
  return v;
}
// block-wide sum / max through shared memory (blockDim.x a multiple of 32, at most 1024); every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* sh) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) sh[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < nw; ++w) t += sh[w];  // fixed order
  return t;
}

__device__ __forceinline__ int row_position(const RowMap& r, int t) { return r.row_pos ? r.row_pos[t] : *r.pos_dev + t; }
__device__ __forceinline__ int row_sequence(const RowMap& r, int t) { return r.row_seq ? r.row_seq[t] : 0; }

// The element-wise kernels of the walk are launched with programmatic stream serialization: a kernel may be placed on
// the SMs while its predecessor still runs, so its launch latency overlaps the predecessor's execution.  Each kernel
// therefore waits for its predecessor (and everything before it) before it reads anything, and lets its successor be
// placed right away; the matrix kernels that follow use that to prefetch weights.
__device__ __forceinline__ void pdl_enter() {
  asm volatile("griddepcontrol.wait;" ::: "memory");
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

constexpr int ATT_THREADS = 256;
constexpr int ATT_MAX_GQA = 8;

// Attention of one row over the keys [s0, s1) of its own list of visible keys, for gqa query heads that share them.
// KV says where key s and value s lie (k(s): dk floats, v(s): dv floats) and what a dot product becomes:
// score(g, s, q_g . k_s).
// sq: the row's query heads of this kv head [gqa][dk] in shared memory (filled and synchronized by the caller);
// sc: [max(gqa * max_chunk, P * gqa * dv)] floats of shared memory, P = max(1, ATT_THREADS / dv); out: the slice's record
// of this row, per query head dv sums, the maximum, the sum of exponentials.
// Ends with the block's threads past their last read of sq and sc only after the caller's next __syncthreads().
template <int ATT_MAX_VALUE, typename KV>  // ATT_MAX_VALUE: the longest value row, a multiple of ATT_THREADS
__device__ __forceinline__ void attend_slice(const KV& src, const float* sq, float* sc, float* out, int s0, int s1, int max_chunk,
                                             int dk, int dv, int gqa) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = ATT_THREADS / 32;
  // scores: one warp per position, all query heads of the group against one read of the K row.  Four positions are in
  // flight per warp (their K rows are fetched before any of them is used): the loop is bound by memory latency, not
  // by arithmetic.  Each position's sum is formed exactly as if it were alone: columns in ascending order per lane.
  constexpr int SP = 4;
  for (int sbase = s0 + warp; sbase < s1; sbase += nw * SP) {
    float acc[SP][ATT_MAX_GQA];
    const float* krow[SP];
#pragma unroll
    for (int j = 0; j < SP; ++j) {
      const int sj = sbase + j * nw;
      krow[j] = sj < s1 ? src.k(sj) : nullptr;
#pragma unroll
      for (int g = 0; g < ATT_MAX_GQA; ++g) acc[j][g] = 0.f;
    }
    for (int i0 = 0; i0 < dk; i0 += 128) {
      float kvv[SP][4];
#pragma unroll
      for (int j = 0; j < SP; ++j)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int i = i0 + lane + 32 * u;
          kvv[j][u] = (krow[j] && i < dk) ? krow[j][i] : 0.f;
        }
#pragma unroll
      for (int j = 0; j < SP; ++j)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int i = i0 + lane + 32 * u;
          if (krow[j] && i < dk) {
#pragma unroll
            for (int g = 0; g < ATT_MAX_GQA; ++g)
              if (g < gqa) acc[j][g] = fmaf(sq[g * dk + i], kvv[j][u], acc[j][g]);
          }
        }
    }
#pragma unroll
    for (int j = 0; j < SP; ++j) {
      const int sj = sbase + j * nw;
      if (sj < s1) {  // warp-uniform
#pragma unroll
        for (int g = 0; g < ATT_MAX_GQA; ++g)
          if (g < gqa) {
            const float d = warp_sum(acc[j][g]);
            if (lane == 0) sc[g * max_chunk + (sj - s0)] = src.score(g, sj, d);
          }
      }
    }
  }
  __syncthreads();
  // per query head: the slice's maximum and the sum of exp(score - max); one warp per head, lanes add in a fixed tree
  for (int g = warp; g < gqa; g += nw) {
    float m = -CUDART_INF_F;
    for (int s = lane; s < s1 - s0; s += 32) m = fmaxf(m, sc[g * max_chunk + s]);
    m = warp_max(m);
    float l = 0.f;
    for (int s = lane; s < s1 - s0; s += 32) {
      const float e = expf(sc[g * max_chunk + s] - m);
      sc[g * max_chunk + s] = e;
      l += e;
    }
    l = warp_sum(l);
    if (lane == 0) { out[g * (dv + 2) + dv] = m; out[g * (dv + 2) + dv + 1] = l; }
  }
  __syncthreads();
  // weighted values: thread (i, grp) owns dimension i (and i + ATT_THREADS, ... where a value row is longer) for every
  // P-th run of eight positions of the slice (P = ATT_THREADS / dv thread groups); the groups' sums are added in group
  // order through shared memory, which the scores leave once every dimension has been summed
  const int P = ATT_THREADS / dv > 0 ? ATT_THREADS / dv : 1;
  const int i = P > 1 || dv == ATT_THREADS ? threadIdx.x % dv : threadIdx.x, grp = P > 1 || dv == ATT_THREADS ? threadIdx.x / dv : 0;
  constexpr int ND = ATT_MAX_VALUE / ATT_THREADS;  // dimensions a thread may own
  float acc[ND][ATT_MAX_GQA];
#pragma unroll
  for (int n = 0; n < ND; ++n)
#pragma unroll
    for (int g = 0; g < ATT_MAX_GQA; ++g) acc[n][g] = 0.f;
  if (grp < P) {
    // runs of eight positions go to the groups in turn: the split does not depend on the KV block size.  The eight
    // value rows of a run are fetched before the first is used; the sums are formed in ascending position order.
    for (int sb = s0 + 8 * grp; sb < s1; sb += 8 * P) {
      float vv[ND][8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float* vrow = sb + j < s1 ? src.v(sb + j) : nullptr;
#pragma unroll
        for (int n = 0; n < ND; ++n) vv[n][j] = vrow && i + n * ATT_THREADS < dv ? vrow[i + n * ATT_THREADS] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (sb + j < s1) {
#pragma unroll
          for (int g = 0; g < ATT_MAX_GQA; ++g)
            if (g < gqa) {
              const float e = sc[g * max_chunk + (sb + j - s0)];
#pragma unroll
              for (int n = 0; n < ND; ++n) acc[n][g] = fmaf(e, vv[n][j], acc[n][g]);
            }
        }
    }
  }
  __syncthreads();  // the scores are no longer needed: their space takes the groups' partial sums
  float* vsum = sc;  // [P][gqa][dv]
#pragma unroll
  for (int n = 0; n < ND; ++n)
    if (grp < P && i + n * ATT_THREADS < dv)
#pragma unroll
      for (int g = 0; g < ATT_MAX_GQA; ++g)
        if (g < gqa) vsum[(grp * gqa + g) * dv + i + n * ATT_THREADS] = acc[n][g];
  __syncthreads();
  for (int idx = threadIdx.x; idx < gqa * dv; idx += ATT_THREADS) {
    float v = 0.f;
    for (int p = 0; p < P; ++p) v += vsum[p * gqa * dv + idx];
    out[(idx / dv) * (dv + 2) + idx % dv] = v;
  }
}

// LLR_WALK_PDL=0 launches these kernels in plain stream order
bool walk_pdl() {
  static const bool on = [] { const char* v = std::getenv("LLR_WALK_PDL"); return !(v && v[0] == '0'); }();
  return on;
}
template <typename... P, typename... A>
cudaError_t launch_walk(void (*kern)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, A... args) {
  cudaLaunchAttribute attr;
  attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr.val.programmaticStreamSerializationAllowed = 1;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cfg.attrs = &attr;
  cfg.numAttrs = walk_pdl() ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, static_cast<P>(args)...);
}

}  // namespace
}  // namespace llr
