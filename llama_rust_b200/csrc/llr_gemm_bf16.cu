// Matrix products with bfloat16 weights for many activation rows on the 5th-generation tensor cores: both operands come
// through TMA into 128-byte swizzled shared memory, tcgen05.mma accumulates in tensor memory (f32), the epilogue reads the
// accumulators with tcgen05.ld.
//
//   y[t][z * rows + r] = sum_c W[z * rows + r][c] * x[t][z * xk + c]        z < batch
//
// With batch 1 this is the chunk form of gemm_f32_x for BF16 weights (langtax/src/quant.rs:6144, :6760); with more it is
// a product per head (a head's rows of W against that head's slice of the activation row).  Activations are bfloat16
// rows (x16); results are f32, or bfloat16 for the product that follows, optionally multiplied by the sigmoid of a
// per-head gate.
//
// With `glu` W stacks gate | up (2 rows rows) and the results are gated units: a tile then holds as many gate rows
// as up rows, so that a thread of the epilogue has both factors of each result.
//
// One CTA computes a tile of 128 activation rows x bn <= BN weight rows: the activation rows are the MMA's M dimension (one
// tensor-memory lane each), so that a thread of the epilogue holds consecutive results of one activation row and stores
// them as vectors.  Six warps: four read the accumulators, one issues the TMA loads, one the MMAs.  Two CTAs fit an SM
// at BN <= 128 (96 KB of stages, 128 columns of tensor memory each), so one tile's epilogue overlaps another's loads.
// bn is the width, a multiple of sixteen, for which the grid's waves over the SMs cost least.  A K range may be cut into slices (gridDim.z): slice s leaves its partial sums at y + s * slice_stride and the reader
// adds them in slice order.  Every wait is bounded.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>

#include "llr_formats.cuh"
#include "llr_kernels.cuh"
#include "llr_tmap.cuh"

namespace llr {
namespace {

constexpr int BM = 128;  // activation rows per CTA = UMMA M
constexpr int BK = 64;   // columns per stage: one 128-byte swizzle row
constexpr int THREADS = 6 * 32, W_TMA = 4, W_MMA = 5;
constexpr int SPIN = 1 << 24;

template <int BN> struct Lay {
  static constexpr int A_STAGE = BM * 128, B_STAGE = BN * 128, STAGE = A_STAGE + B_STAGE;
  static constexpr int NS = BN == 256 ? 4 : BN == 128 ? 3 : 4;  // 192, 96, 96 KB
  static constexpr int BAR = NS * STAGE;
  static constexpr int TOTAL = 1024 /*alignment*/ + NS * STAGE + 256;
  static constexpr int TMEM_COLS = BN;
};

__device__ __forceinline__ uint32_t s32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void bar_init(uint64_t* b, int n) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(s32(b)), "r"(n) : "memory");
}
__device__ __forceinline__ void bar_expect(uint64_t* b, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(s32(b)), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool bar_wait(uint64_t* b, uint32_t parity) {
  for (int spins = 0; spins < SPIN; ++spins) {
    uint32_t ok;
    asm volatile("{ .reg .pred p; mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2; selp.u32 %0, 1, 0, p; }"
                 : "=r"(ok) : "r"(s32(b)), "r"(parity) : "memory");
    if (ok) return true;
  }
  return false;
}
__device__ __forceinline__ bool elect_one() {
  uint32_t pred;
  asm volatile("{ .reg .pred p; elect.sync _|p, 0xffffffff; selp.u32 %0, 1, 0, p; }" : "=r"(pred));
  return pred != 0;
}
// K-major operand tile of 128-byte swizzled rows: eight-row groups 1024 bytes apart (as in llr_gemm_tc.cu)
__device__ __forceinline__ uint64_t tile_desc(uint32_t saddr) {
  return ((uint64_t)(saddr >> 4) & 0x3fffu) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
// kind::f16: f32 accumulator, both operands bfloat16, M = 128, N = bn
__device__ __forceinline__ uint32_t mma_desc(int bn) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(bn >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
}

struct Args {
  float* y;
  __nv_bfloat16* y16;
  const float* gate;   // gate[t * gate_ld + z]: results times its sigmoid
  int64_t y_ld, gate_ld, slice_stride;
  int tokens, rows, nk, xk;  // nk: 64-column steps of the whole K range
  int batch, slices, bn;
  GluShape glu;
};

// 32 accumulator columns of this warp's 32 lanes
__device__ __forceinline__ void load32(uint32_t taddr, uint32_t (&v)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
      "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
        "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
        "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
        "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
      : "r"(taddr) : "memory");
}

template <int BN, bool GLU>
__global__ void __launch_bounds__(THREADS)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap xmap, const __grid_constant__ CUtensorMap wmap, const Args a, int* __restrict__ err) {
  using L = Lay<BN>;
  constexpr int NS = L::NS;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint64_t* full = (uint64_t*)(smem + L::BAR);
  uint64_t* empty = full + NS;
  uint64_t* done = empty + NS;
  uint32_t* tmem_slot = (uint32_t*)(done + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int bn = a.bn, width = GLU ? bn / 2 : bn;  // results per activation row of the tile
  // token tiles run fastest: the CTAs that share weight rows run at the same time, and the weights are read from HBM once
  const int row0 = blockIdx.y * width, tok0 = blockIdx.x * BM;
  const int z = (int)blockIdx.z / a.slices, slice = (int)blockIdx.z % a.slices;
  const int per = (a.nk + a.slices - 1) / a.slices, k0 = slice * per, k1 = min(a.nk, k0 + per);  // never empty: the launcher sees to it

  if (threadIdx.x == 0) {
    for (int s = 0; s < NS; ++s) { bar_init(&full[s], 1); bar_init(&empty[s], 1); }
    bar_init(done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == W_MMA) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(s32(tmem_slot)), "r"(L::TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *tmem_slot;
  bool ok = true;

  if (warp == W_TMA) {
    const uint32_t base = __shfl_sync(0xffffffffu, s32(smem), 0);
    for (int k = k0; k < k1; ++k) {
      const int s = (k - k0) % NS;
      if (ok && !bar_wait(&empty[s], (uint32_t)((((k - k0) / NS) & 1) ^ 1))) { ok = false; report_error(err, 5); }
      if (ok && elect_one()) {
        bar_expect(&full[s], (uint32_t)(L::A_STAGE + bn * 128));  // boxes are always complete: what lies outside the matrices is filled with zeros
        asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                     ::"r"(base + (uint32_t)(s * L::STAGE + L::A_STAGE)), "l"(&wmap), "r"(k * BK), "r"(z * a.rows + row0), "r"(s32(&full[s])) : "memory");
        if constexpr (GLU)
          asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                       ::"r"(base + (uint32_t)(s * L::STAGE + L::A_STAGE + width * 128)), "l"(&wmap), "r"(k * BK), "r"(a.rows + row0), "r"(s32(&full[s])) : "memory");
        asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                     ::"r"(base + (uint32_t)(s * L::STAGE)), "l"(&xmap), "r"(z * a.xk + k * BK), "r"(tok0), "r"(s32(&full[s])) : "memory");
      }
      __syncwarp();
    }
  } else if (warp == W_MMA) {
    const uint32_t idesc = mma_desc(bn);
    const uint32_t td = __shfl_sync(0xffffffffu, tmem, 0), base = __shfl_sync(0xffffffffu, s32(smem), 0);
    for (int k = k0; k < k1; ++k) {
      const int s = (k - k0) % NS;
      if (ok && !bar_wait(&full[s], (uint32_t)(((k - k0) / NS) & 1))) { ok = false; report_error(err, 5); }
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      if (elect_one()) {
        const uint64_t da = tile_desc(base + (uint32_t)(s * L::STAGE)), db = tile_desc(base + (uint32_t)(s * L::STAGE + L::A_STAGE));
#pragma unroll
        for (int kk = 0; kk < BK / 16; ++kk) {
          const uint32_t acc = (k > k0 || kk > 0) ? 1u : 0u;
          asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0; tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }"
                       ::"r"(td), "l"(da + 2 * kk), "l"(db + 2 * kk), "r"(idesc), "r"(acc) : "memory");
        }
        asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(s32(&empty[s])) : "memory");
      }
      __syncwarp();
    }
    if (elect_one())
      asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(s32(done)) : "memory");
    __syncwarp();
  } else {
    if (!bar_wait(done, 0)) { ok = false; report_error(err, 5); }
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const int t = tok0 + 32 * warp + lane;
    const int n_live = min(width, a.rows - row0);
    const int64_t off = (int64_t)t * a.y_ld + (int64_t)z * a.rows + row0;
    float* y = a.y ? a.y + slice * a.slice_stride + off : nullptr;
    __nv_bfloat16* y16 = a.y16 ? a.y16 + off : nullptr;
    float gate = 1.f;
    if (a.gate && t < a.tokens) gate = 1.0f / (1.0f + expf(-a.gate[(int64_t)t * a.gate_ld + z]));
    const bool vec = ((a.y_ld | a.rows) & 7) == 0;  // every run of eight results starts on a 16-byte boundary in either format
#pragma unroll 1
    for (int c0 = 0; c0 < n_live; c0 += 32) {
      uint32_t v[32], u[32];
      const uint32_t taddr = tmem + ((uint32_t)(32 * warp) << 16) + (uint32_t)c0;
      load32(taddr, v);
      if constexpr (GLU) load32(taddr + (uint32_t)width, u);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      if (t < a.tokens) {
        float f[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          if constexpr (GLU) f[j] = gated_unit(__uint_as_float(v[j]), __uint_as_float(u[j]), a.glu);
          else f[j] = a.gate ? __uint_as_float(v[j]) * gate : __uint_as_float(v[j]);
        }
        if (vec) {
#pragma unroll
          for (int j = 0; j < 32; j += 8)
            if (c0 + j < n_live) {  // rows is a multiple of eight here
              if (y) {
                *(float4*)(y + c0 + j) = make_float4(f[j], f[j + 1], f[j + 2], f[j + 3]);
                *(float4*)(y + c0 + j + 4) = make_float4(f[j + 4], f[j + 5], f[j + 6], f[j + 7]);
              }
              if (y16) {
                __nv_bfloat162 h[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) h[u] = __floats2bfloat162_rn(f[j + 2 * u], f[j + 2 * u + 1]);
                *(uint4*)(y16 + c0 + j) = *(const uint4*)h;
              }
            }
        } else {
#pragma unroll
          for (int j = 0; j < 32; ++j)
            if (c0 + j < n_live) {
              if (y) y[c0 + j] = f[j];
              if (y16) y16[c0 + j] = __float2bfloat16_rn(f[j]);
            }
        }
      }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  }
  __syncthreads();
  if (warp == W_MMA) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(L::TMEM_COLS) : "memory");
  }
}

bool encode_rows(CUtensorMap* map, const void* base, int64_t cols, int64_t rows, int64_t ld, int box_rows) {
  EncodeTiledFn enc = tensor_map_encoder();
  if (!enc) return false;
  const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {(cuuint32_t)BK, (cuuint32_t)box_rows};
  const cuuint32_t one[2] = {1, 1};
  return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void*)base, dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN, bool GLU>
cudaError_t launch_tiles(const Bf16Product& p, const Args& a, cudaStream_t stream, int* err) {
  CUtensorMap xmap, wmap;
  const int width = GLU ? a.bn / 2 : a.bn;  // rows of one box of W
  if (!encode_rows(&xmap, p.x16, p.x_cols, p.tokens, p.x_ld, BM) || !encode_rows(&wmap, p.w, p.cols, (int64_t)p.rows * (GLU ? 2 : p.batch), p.cols, width))
    return cudaErrorInvalidValue;
  constexpr int smem = Lay<BN>::TOTAL;
  static PerDevice ready;
  std::atomic<int>& slot = ready.here();
  if (slot.load(std::memory_order_relaxed) == 0) {
    const cudaError_t e = cudaFuncSetAttribute(gemm_bf16_kernel<BN, GLU>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    slot.store(1, std::memory_order_relaxed);
  }
  const dim3 grid((unsigned)((p.tokens + BM - 1) / BM), (unsigned)((p.rows + width - 1) / width), (unsigned)(p.batch * a.slices));
  if (grid.y > 65535 || grid.z > 65535) return cudaErrorInvalidValue;
  gemm_bf16_kernel<BN, GLU><<<grid, THREADS, smem, stream>>>(xmap, wmap, a, err);
  return cudaGetLastError();
}

constexpr int SMS = 148;
int tiles_of(int tokens, int rows, int batch, int bn) { return ((tokens + BM - 1) / BM) * ((rows + bn - 1) / bn) * batch; }
// Width of a tile: with many tiles the one of 160 .. 256 (a multiple of `step`, so that both halves of a gated tile are
// whole eight-row groups) whose waves over the SMs cost least, where a wave costs as much as its columns and WAVE_COST
// more (measured: it hardly depends on the width); otherwise 128 or 64.
constexpr int WAVE_COST = 450;
int tile_width(int tokens, int rows, int batch, int step = 16) {
  if (tiles_of(tokens, rows, batch, 256) < 132) return rows > 64 ? 128 : 64;
  int best = 256, cost = 1 << 30;
  for (int bn = 256; bn >= 160; bn -= step) {
    const int c = (tiles_of(tokens, rows, batch, bn) + SMS - 1) / SMS * (bn + WAVE_COST);
    if (c < cost) { cost = c; best = bn; }
  }
  return best;
}

}  // namespace

bool gemm_bf16_supported(const void* w, int64_t rows, int64_t cols) {
  return rows > 0 && rows < (1 << 28) && cols > 0 && cols < (1 << 28) && cols % 8 == 0 && ((uintptr_t)w & 15) == 0;
}

// K slices of a product without heads: as many as keep the grid within one wave of two CTAs per SM, every slice at
// least 512 columns long
int gemm_bf16_slices(int tokens, int rows, int cols) {
  const int bn = tile_width(tokens, rows, 1);
  if (bn > 128) return 1;
  const int tiles = tiles_of(tokens, rows, 1, bn), nk = (cols + BK - 1) / BK;
  int s = 1;
  while (s < 8 && tiles * s * 2 <= 296 && nk / (s * 2) >= 8) s *= 2;
  while (s > 1 && (s - 1) * ((nk + s - 1) / s) >= nk) s /= 2;  // no empty slice
  return s;
}

cudaError_t launch_gemm_bf16(const Bf16Product& p, cudaStream_t stream, int* err, uint64_t* launches) {
  if (p.tokens <= 0) return cudaSuccess;
  if (!gemm_bf16_supported(p.w, p.rows, p.cols) || p.batch < 1 || p.x_ld % 8 != 0 || (p.batch > 1 && p.xk % 8 != 0) || ((uintptr_t)p.x16 & 15) != 0 ||
      (((uintptr_t)p.y | (uintptr_t)p.y16) & 15) != 0 || p.slices < 1 || (p.slices > 1 && (p.batch != 1 || p.y16 || p.gate || p.glu)) ||
      (p.glu && (p.batch != 1 || p.gate)))
    return cudaErrorInvalidValue;
  Args a{};
  a.y = p.y; a.y16 = (__nv_bfloat16*)p.y16; a.gate = p.gate;
  a.y_ld = p.y_ld; a.gate_ld = p.gate_ld; a.slice_stride = p.slice_stride;
  a.tokens = p.tokens; a.rows = p.rows; a.nk = (p.cols + BK - 1) / BK; a.xk = p.xk;
  a.batch = p.batch; a.slices = p.slices;
  if ((a.slices - 1) * ((a.nk + a.slices - 1) / a.slices) >= a.nk) return cudaErrorInvalidValue;
  if (launches) ++*launches;
  if (p.glu) {
    a.glu = *p.glu;
    a.bn = std::max(tile_width(p.tokens, 2 * p.rows, 1, 32), 128);
    return a.bn > 128 ? launch_tiles<256, true>(p, a, stream, err) : launch_tiles<128, true>(p, a, stream, err);
  }
  a.bn = tile_width(p.tokens, p.rows, p.batch);
  if (a.bn > 128) return launch_tiles<256, false>(p, a, stream, err);
  return a.bn == 128 ? launch_tiles<128, false>(p, a, stream, err) : launch_tiles<64, false>(p, a, stream, err);
}

}  // namespace llr
