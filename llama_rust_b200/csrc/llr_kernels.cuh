// Internal launch interface between the executor (llr_exec.cu) and the kernels.
#pragma once
#include <cuda_runtime.h>
#include <stddef.h>
#include <stdint.h>

#include <atomic>
#include <string>
#include <vector>

namespace llr {

// One-time setup of a kernel, per device: function attributes and occupancy belong to a device's context, and executors
// of several devices (and threads) may share a process.  here() is the current device's slot; 0 means not set up yet
// (two threads that both find 0 do the same setup and store the same value).
struct PerDevice {
  std::atomic<int> slot[64];
  std::atomic<int>& here() {
    int d = 0;
    cudaGetDevice(&d);
    return slot[d & 63];
  }
};

// A resident packed matrix as the kernels see it.  `w` is 256-byte aligned and
// the allocation is padded so that 16-byte windows around any row are readable.
// Error word of an executor: one int in mapped pinned host memory.  A kernel whose bounded wait
// ran out stores a non-zero code with a plain store (any writer wins); the host reads the word
// after synchronizing, with no copy on the path.
#ifdef __CUDACC__
__device__ __forceinline__ void report_error(int* err, int code) { *(volatile int*)err = code; }
#endif

struct MatView {
  const uint8_t* w;
  int dtype;
  int64_t rows, cols;
  int64_t row_bytes;
  int f16_ok = -1;  // tensor-core GEMM operand choice: 1 binary16 (weights fit its range), 0 bfloat16, -1 not examined (bfloat16)
};

enum GemvPath : int { PATH_AUTO = 0, PATH_GENERIC = 1, PATH_STAGED = 2, PATH_MMA = 3, PATH_TC = 4 };
constexpr int64_t TC_MIN_TOKENS = 64;  // from here on AUTO prefers the bf16 tcgen05 GEMM

// y[t*rows + r] = sum_c W[r,c] * x[t*cols + c] for t < tokens.  Any shape the
// entry points accept.  `launches` is incremented by the kernels launched.
// `err_flag` is a device int that kernels with bounded waits set to non-zero when a wait ran out.
// `scratch` (matmul_scratch_bytes, or null) lets the tensor-core GEMM stage 16-bit activations.
cudaError_t launch_matmul(const MatView& m, const float* x, float* y, int64_t tokens,
                          cudaStream_t stream, int path, int sm_count, int* err_flag,
                          void* scratch, uint64_t* launches);
bool matmul_wants_tc(const MatView& m, int64_t tokens, int path);
size_t matmul_scratch_bytes(const MatView& m, int64_t tokens);  // for launch_matmul when matmul_wants_tc

// Always-available reference kernel: one warp per row, byte loads, any alignment.
cudaError_t launch_gemv_generic(const MatView& m, const float* x, float* y, int64_t tokens,
                                cudaStream_t stream, uint64_t* launches);

// Shared-memory staged decode GEMV (tokens <= 8 per pass); see llr_gemv_staged.cu.
bool gemv_staged_supported(const MatView& m);
cudaError_t launch_gemv_staged(const MatView& m, const float* x, float* y, int64_t tokens,
                               cudaStream_t stream, int sm_count, uint64_t* launches);

// Streaming decode GEMV for the element formats F32 / F16 / BF16 (tokens <= 8 per pass); see llr_gemv_rows.cu.
bool gemv_rows_supported(const MatView& m);
cudaError_t launch_gemv_rows(const MatView& m, const float* x, float* y, int64_t tokens, cudaStream_t stream, int sm_count,
                             uint64_t* launches);

struct GluShape;
// A stacked gate | up matrix (2 n rows) and the clamped gated unit of its products in one launch (tokens <= 8): out[t][i]
cudaError_t launch_gemv_rows_glu(const MatView& m, const float* x, float* out, const GluShape& glu, int tokens, cudaStream_t stream,
                                 int sm_count, uint64_t* launches);

// Integer tensor-core decode GEMV for Q4_K / Q6_K / Q8_0 (tokens <= 8 per pass); see
// llr_gemv_stream.cu.  Launched with programmatic stream serialization.
bool gemv_mma_supported(const MatView& m);
cudaError_t launch_gemv_mma(const MatView& m, const float* x, float* y, int64_t tokens,
                            cudaStream_t stream, int sm_count, int* err_flag, uint64_t* launches);
// Result delivery to the host by the kernel itself (host-pointer calls with at most 8 activation
// rows): the reducer also stores each finished value at y + y_delta bytes, a device alias of
// mapped pinned host memory, and the CTA that finishes last stores `ticket` into *done (mapped
// pinned as well) after a system-scope fence.  The host polls *done instead of enqueuing a
// device-to-host copy and synchronizing the stream.  count is a zeroed device word.
struct HostOut {
  long long y_delta;
  int* done;
  unsigned int* count;
  int ticket;
};
// One product with ONE activation row whose matrix a kernel earlier in the stream chooses: the weights are addressed
// through maps_dev[*sel_dev], an array (device memory) of GEMV_MAP_BYTES-byte tensor maps that gemv_mma_encode_map filled
// for matrices of one shape and format (`shape`: any of them).  No host round trip between the choice and the product.
constexpr int GEMV_MAP_BYTES = 128;
cudaError_t gemv_mma_encode_map(const MatView& m, void* map_out);
cudaError_t launch_gemv_mma_select(const MatView& shape, const void* maps_dev, const int* sel_dev, const float* x, float* y,
                                   cudaStream_t stream, int sm_count, int* err_flag, uint64_t* launches);
bool gemv_mma_hostout_ok(const MatView& m, int64_t tokens);
cudaError_t launch_gemv_mma_hostout(const MatView& m, const float* x, float* y, int64_t tokens, const HostOut& ho,
                                    cudaStream_t stream, int sm_count, int* err_flag, uint64_t* launches);

// One matrix product of a program (llr_gemv_stream.cu).  The caller fills the first block and the
// operation fields; tile_begin / n_tiles and everything about tagged buffers are filled in by
// program_create.
//
// Tagged buffers.  A result that a later entry of the same program reads is also written as 8-byte
// pairs {f32 bits, tag}, tag = tag_base of the run + producing phase.  A consumer loads pairs and
// spins (bounded) until every tag is the expected one: the value is its own arrival signal, so no
// counter, fence or poll separates a phase from the next.
enum XOp : int {
  XOP_NONE = 0,     // x as it is
  XOP_RMSNORM = 1,  // x * (1 / sqrt(mean(x^2) + eps)) * x2[c]   (x2: norm weights, plain f32, may be null)
  XOP_SWIGLU = 2,   // silu(x) * x2[c]                            (x2: the `up` vector)
};
struct ProgEntry {
  const uint8_t* w;
  const float* x;     // input, plain f32 (ignored by the kernel when xt is set)
  float* y;           // result, plain f32 (this rank's slice)
  int64_t row_bytes;
  int rows, cols, dtype, tokens;
  int tile_begin, n_tiles;
  int64_t y_ld;  // floats between consecutive activation rows of y (0: rows); larger when y is a slice of a wider vector
  // ---- 64 bytes
  const void* xt;     // tagged input (pairs), or null
  const void* x2;     // second operand of x_op: plain f32, or pairs when x2_phase >= 0
  const void* resid;  // added to the finished result, indexed like y: plain f32, or pairs when resid_phase >= 0; may be null
  void* yt;           // tagged copy of the result (this rank's slice), or null when no entry reads it
  int x_op;
  float eps;
  int x_phase, x2_phase, resid_phase;  // phase that writes the tagged source (-1: plain memory, ready at launch)
  int sel_slot, map_base;  // select programs (program_set_select): the matrix is maps[map_base + sel[sel_slot]]
  int pad;
};
static_assert(sizeof(ProgEntry) == 128, "entries are copied as sixteen 8-byte words");
// Row-sharded programs across GPUs: where the other ranks keep their copies of the results
// and of the phase counters.  peer address = local address + delta[g] bytes (arenas have one layout).
struct PeerTable {
  int n_peers;  // other ranks (world size - 1), at most 7
  int pad;
  unsigned long long* counters[7];
  long long y_delta[7];
};
// wait_prev: bit 0 = wait for the previous phase's counter, bit 1 = publish this phase's counter,
// bit 2 (phase 0 of a sharded program) = wait for the end of the previous run on every rank.
struct ProgPhase { int first_entry, n_entries, n_tiles, wait_prev; };
struct Program;
bool prog_entry_supported(const MatView& m);
// Placement of a sharded program's buffers: the arena is header | result area of result_bytes |
// tagged area of 2 * result_bytes; the pair of the float at result offset o lies at tagged offset 2 o.
struct ShardInfo {
  unsigned long long* counters;  // arena header
  PeerTable peers;
  char* arena;
  size_t result_bytes;
  int world, rank;
};
// phase_of[i] is non-decreasing.  strict_phases: an input that is not an earlier entry's result makes
// its phase wait until the previous phase is completely written (counter per phase); otherwise such
// inputs are read as they are at launch.
cudaError_t program_create(const std::vector<ProgEntry>& entries, const std::vector<int>& phase_of,
                           int sm_count, bool strict_phases, const ShardInfo* shard, Program** out, std::string* msg);
void program_destroy(Program* p);
// Turns a one-phase, one-token program without operations into a select program: entry E then reads its weights through
// maps_dev[E.map_base + sel_dev[E.sel_slot]] (tensor maps of gemv_mma_encode_map, matrices shaped like E) instead of
// E.w.  The table is read on the device when the launch runs, after the kernels before it in the stream.
cudaError_t program_set_select(Program* p, const void* maps_dev, const int* sel_dev);
// poll_limit: iterations a device-side wait for another CTA's or rank's data may take before it gives up
cudaError_t program_run(Program* p, cudaStream_t stream, int* err_flag, int poll_limit, uint64_t* launches);
int program_phases(const Program* p);
int program_entries(const Program* p);
int program_counter_phases(const Program* p);
int program_grid(const Program* p);  // phases that synchronise through a counter

// dequant -> shared memory -> tcgen05/TMEM chunk GEMM (bf16 operands, f32 accumulate) for
// Q4_K / Q8_0 / Q5_0 / Q5_1 with many activation rows; see llr_gemm_tc.cu.
bool gemm_tc_supported(const MatView& m, int64_t tokens);
// Examines the block headers of a matrix the GEMM can take: writes the bit pattern of the largest
// possible |weight| to *out_dev (device); weight_bound_allows_f16 turns that into the operand choice.
cudaError_t launch_weight_bound(const MatView& m, unsigned int* out_dev, cudaStream_t stream, uint64_t* launches);
bool weight_bound_allows_f16(unsigned int bound_bits);
// Grouped launch: several products of one dtype in one grid (routed experts).  x16 / xscale are
// the group's activations as tc_convert_activations left them; desc_dev is device scratch of
// gemm_tc_group_desc_bytes(n) bytes, 64-byte aligned.
struct GemmGroupSpec {
  MatView m;
  const void* x16;
  const float* xscale;
  float* y;
  int tokens;
};
size_t gemm_tc_group_desc_bytes(int n_groups);
cudaError_t tc_convert_activations(const float* x, int64_t n_rows, int cols, bool f16, void* out16, float* xscale,
                                   cudaStream_t stream, uint64_t* launches);
// Routed-expert layer: 16-bit operand row r from row src_row[r] of x (cols a multiple of 4, rows
// 16-byte aligned).
cudaError_t tc_convert_expert_rows(const float* x, const int* src_row, int64_t n_rows, int cols, bool f16,
                                   void* out16, float* xscale, cudaStream_t stream, uint64_t* launches);
cudaError_t launch_gemm_tc_grouped(const GemmGroupSpec* specs, int n_groups, bool f16, void* desc_dev,
                                   cudaStream_t stream, int* err_flag, uint64_t* launches);
size_t gemm_tc_scratch_bytes(const MatView& m, int64_t tokens);
cudaError_t launch_gemm_tc(const MatView& m, const float* x, float* y, int64_t tokens, void* scratch, size_t scratch_bytes,
                           cudaStream_t stream, int* err_flag, uint64_t* launches);

// Same kernels with the staging buffer in a file-scope __device__ array (no allocation).
constexpr size_t GEMM_STATIC_SCRATCH_BYTES = 32u << 20;
size_t gemm_tc_static_scratch_limit();
cudaError_t launch_gemm_tc_static(int device, const MatView& m, const float* x, float* y, int64_t tokens,
                                  cudaStream_t stream, int* err_flag, uint64_t* launches);

// Routed-expert FFN glue (llr_moe.cu)
cudaError_t launch_gather_rows(const float* x, const int* tok_of_row, float* packed, int n_rows, int n_embd,
                               cudaStream_t s, uint64_t* launches);
cudaError_t launch_silu_mul(float* g, const float* u, int64_t n, cudaStream_t s, uint64_t* launches);
// logits[t*n_expert + e] = dot(w[e], x[t]) for an F32 router matrix (n_embd % 4 == 0, 16-byte aligned)
cudaError_t launch_router_logits(const float* w, const float* x, float* logits, int tokens, int n_expert, int n_embd,
                                 cudaStream_t s, uint64_t* launches);
// Routing on the device: softmax / top-k / weights per token in place on the logits, then the packed row order
cudaError_t launch_route(float* logits, int tokens, int n_expert, int n_used, int norm_w, int* ids, float* wts,
                         cudaStream_t s, uint64_t* launches);
cudaError_t launch_bucket(const int* ids, const float* wts, const unsigned char* local, int tokens, int n_expert, int n_used,
                          int* first_row, int* tok_of_row, int* rows_of_tok, float* w_of_tok, int* fill, cudaStream_t s,
                          uint64_t* launches);
cudaError_t launch_scatter_combine(const float* y, const int* rows_of_tok, const float* w_of_tok, float* out,
                                   int tokens, int n_used, int n_embd, cudaStream_t s, uint64_t* launches);
// One token without a host round trip: its selection sorted by expert id (n_used <= 8), and the combine of its experts' rows
cudaError_t launch_select_sorted(const int* ids, const float* wts, int n_used, int* sel, float* selw, cudaStream_t s, uint64_t* launches);
cudaError_t launch_combine_one(const float* y, const float* selw, float* out, int n_used, int n_embd, cudaStream_t s, uint64_t* launches);

// Expert parallelism over peer stores (llr_moe_ep.cu).  An arena starts with an EpHeader, then twice (runs
// alternate): counts [local expert][sender], packed row numbers and rows [local expert][sender][t_max], and the
// return area [t_max * n_used] rows.
constexpr int EP_MAX_WORLD = 8;
struct EpHeader {
  unsigned long long flag_in[EP_MAX_WORLD];    // [sender]: last run whose rows from that sender are complete here
  unsigned long long flag_back[EP_MAX_WORLD];  // [owner]: last run whose results from that owner are complete here
  unsigned long long done_dispatch, done_return;  // this rank's CTAs, counted over all runs
};
struct EpPeers { char* arena[EP_MAX_WORLD]; };  // every rank's arena as mapped here (entry `rank`: this rank's own)
struct EpLayout {
  int n_expert, n_used, n_embd, world, rank, t_max, e_loc;
  size_t cnt_off[2], tag_off[2], recv_off[2], back_off[2], total;
};
EpLayout ep_layout(int n_expert, int n_used, int n_embd, int world, int rank, int t_max);
cudaError_t launch_ep_dispatch(const float* x, const int* tok_of_row, const int* first_row, int n_rows, const EpPeers& peers,
                               const EpLayout& L, int parity, unsigned long long epoch, unsigned long long done_target,
                               cudaStream_t s, uint64_t* launches);
cudaError_t launch_ep_wait(const unsigned long long* flags, int world, unsigned long long epoch, int poll_limit, int* err,
                           cudaStream_t s, uint64_t* launches);
cudaError_t launch_ep_gather(const char* arena, const EpLayout& L, int parity, const int* seg_first, int n_seg, int n_rows,
                             float* rows, int* ret_src, int* ret_tag, cudaStream_t s, uint64_t* launches);
cudaError_t launch_ep_return(const float* y, const int* ret_src, const int* ret_tag, int n_rows, const EpPeers& peers,
                             const EpLayout& L, int parity, unsigned long long epoch, unsigned long long done_target,
                             cudaStream_t s, uint64_t* launches);

// out[(r-row0)*cols + c] = dequantized W[r,c], bit-exact with the reference.
cudaError_t launch_dequant(const MatView& m, int64_t row0, int64_t n_rows, float* out,
                           cudaStream_t stream, uint64_t* launches);

// out[i*cols + c] = dequantized W[ids[i], c] with ids in device memory (token embeddings)
cudaError_t launch_dequant_indexed(const MatView& m, const int* ids_dev, int64_t n, float* out,
                                   cudaStream_t stream, uint64_t* launches);

// ---- element-wise and attention kernels of the device-resident Llama walk (llr_decode.cu) ----
struct WalkShape { int n_embd, n_head, n_head_kv, head_dim, n_ff, n_ctx; float rms_eps, rope_base, theta_scale; };
// y[t] = (x[t] * 1/sqrt(mean(x[t]^2) + eps)) * w; with `add` non-null first x[t] += add[t] (written back: the new
// residual stream).  w may be null (all ones).
cudaError_t launch_rmsnorm(float* x, const float* add, const float* w, float* y, int tokens, int n, float eps,
                           cudaStream_t s, uint64_t* launches);
// Paged KV cache as the kernels see it (langtax/src/kv_page.rs:395-437: a head vector of block b lies at
// (((b * n_layers + layer) * n_head_kv + head) * block_tokens + t % block_tokens) * head_dim, b = table[t / block_tokens]).
// table holds max_blocks entries per sequence.
struct KvView {
  float* k;
  float* v;
  const int* table;
  int block_tokens, max_blocks, n_layer;
};
// Where the rows of a batch stand: row t belongs to sequence row_seq[t] at position row_pos[t]; with null arrays all
// rows belong to sequence 0 at positions *pos_dev + t (the position counter lives in device memory so that a captured
// or pre-enqueued step sees the current value).
struct RowMap {
  const int* pos_dev;
  const int* row_pos;
  const int* row_seq;
};
// RoPE (adjacent pairs) on q and k at each row's position, then k and v into the cache.
cudaError_t launch_rope_store(float* q, float* k, const float* v, const KvView& kv, const RowMap& rows, int tokens, int layer,
                              const WalkShape& w, cudaStream_t s, uint64_t* launches);
// out[t][hq] = softmax(q[t][hq] . K[0..pos(t)] / sqrt(hd)) V over row t's own sequence, grouped-query heads; scratch holds
// the partial results of the position splits (attention_scratch_floats)
size_t attention_scratch_floats(int tokens, const WalkShape& w);
cudaError_t launch_attention(const float* q, const KvView& kv, float* out, float* scratch, const RowMap& rows, int tokens,
                             int layer, const WalkShape& w, cudaStream_t s, uint64_t* launches,
                             const float* k_new = nullptr, const float* v_new = nullptr,  // k_new / v_new: one decode token whose rotation and cache store the attention kernel does itself
                             bool tensor_cores = false,  // a prompt chunk of one sequence may run as binary16 MMAs with f32 accumulation (the tolerance of the 16-bit chunk GEMM)
                             bool one_sequence = false);  // the caller vouches that the rows are one sequence at consecutive positions (rows given per row)
cudaError_t launch_swiglu(float* g, const float* u, int64_t n, cudaStream_t s, uint64_t* launches);
cudaError_t launch_add(float* x, const float* y, int64_t n, cudaStream_t s, uint64_t* launches);
// first index of the strict maximum of logits[0..n) -> *out_id (device; n == 0: no argmax), and *pos_dev += advance
// With count_dev the token also goes to out_id[1 + *count_dev], its margin to out_margin[*count_dev], and the
// count grows by one (a generation loop whose steps are identical launches).
// part: 384 words of device scratch (a long row is scanned by many blocks), or null
cudaError_t launch_argmax_advance(const float* logits, int n, int* out_id, float* out_margin, int* pos_dev, int advance,
                                  int* count_dev, float* part, cudaStream_t s, uint64_t* launches);
// one argmax per row of logits[n_rows][n] -> out_id[row], out_margin[row] (optional)
cudaError_t launch_argmax_rows(const float* logits, int n_rows, int n, int* out_id, float* out_margin, cudaStream_t s,
                               uint64_t* launches);

// Gated unit of n results.  UNIT_CLAMPED: a * sigmoid(alpha * a) * (b + shift), a = min(gate, limit), b = clamp(up, -limit,
// limit).  UNIT_GELU: gelu(gate) * up with the tanh form of gelu.
enum GatedUnit : int { UNIT_CLAMPED = 0, UNIT_GELU = 1 };
struct GluShape { int n; float limit, alpha, shift; int unit; };
#ifdef __CUDACC__
// 0.5 z (1 + tanh(w)) = z sigmoid(2 w), w = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh(float z) {
  const float w2 = __fmul_rn(1.5957691216057308f, __fmul_rn(z, fmaf(0.044715f, __fmul_rn(z, z), 1.0f)));
  return __fdiv_rn(z, 1.0f + expf(-w2));
}
__device__ __forceinline__ float gated_unit(float a, float b, const GluShape& g) {
  if (g.unit == UNIT_GELU) return __fmul_rn(gelu_tanh(a), b);
  a = fminf(a, g.limit);
  b = fminf(fmaxf(b, -g.limit), g.limit);
  return __fmul_rn(__fmul_rn(a, __fdiv_rn(1.0f, 1.0f + expf(-__fmul_rn(g.alpha, a)))), __fadd_rn(b, g.shift));
}
#endif
// ---- products with bfloat16 weights for many rows (llr_gemm_bf16.cu): tcgen05, bfloat16 activations, f32 accumulation ----
// y[t * y_ld + z * rows + r] = sum_c W[z * rows + r][c] x[t][z * xk + c] for z < batch (a product per head), times
// sigmoid(gate[t * gate_ld + z]) when gate is set.  Results as f32 (y), as bfloat16 (y16), or both.  With slices > 1
// (batch 1, y only) slice s of the K range leaves its partial sums at y + s * slice_stride.
struct Bf16Product {
  const void* w;      // [batch * rows][cols]
  const void* x16;    // [tokens][x_ld], of which x_cols columns exist
  int64_t x_ld, x_cols;
  float* y;
  void* y16;
  const float* gate;
  int64_t y_ld, gate_ld, slice_stride;
  int tokens, rows, cols, batch, xk, slices;
  const GluShape* glu;  // W stacks gate | up, 2 rows rows: the results are gated units (batch 1)
};
bool gemm_bf16_supported(const void* w, int64_t rows, int64_t cols);
int gemm_bf16_slices(int tokens, int rows, int cols);
cudaError_t launch_gemm_bf16(const Bf16Product& p, cudaStream_t stream, int* err, uint64_t* launches);
constexpr int BF16_TC_MIN_TOKENS = 16;  // from here on the walk of a layered decoder prefers it

// ---- kernels of decoders described layer by layer (llr_mixers.cu) ----
// A layer's keys and values in the paged pool: head vector of (block b, kv head g, position t of the block) lies at
// k + b * k_block + (g * block_tokens + t) * dk, values likewise; a latent layer has one vector per position that serves
// as key and value of every head (v == k).
struct LayerKv {
  float* k;
  float* v;
  const int* table;
  int block_tokens, max_blocks;
  int64_t k_block, v_block;
};
// What a row attends to and how it scores: n_head query heads over n_kv key/value heads (n_head / n_kv share one), the
// last `window` positions (0: all) and the first keep_first; score = (q . k) * scale + bias[h][min(distance, bias_len - 1)].
// sink[h] (may be null) is one more score that has no value: exp(sink) stands in the denominator.
struct SpanShape {
  int n_head, n_kv, dk, dv, window, keep_first, n_ctx;
  float scale;
  const float* bias;  // [n_head][bias_len], or null
  int bias_len;
  const float* sink;  // [n_head], or null
};
// Rotation of a head's first dims values, pairs (i, i + dims / 2): row t's cosines and sines are the dims / 2 entries from
// cs + t * ld on.  dims 0: none.
struct RotRows {
  const float2* cs;
  int ld, dims;
};
// Every distinct rotation of a model, end to end: cs[t * n + i] = (cos, sin)(position of t * freq[i])
struct RotTable {
  const double* freq;
  float2* cs;
  int n;
};
// x[t] = table[ids[t]] * scale + pos_table[position of t]; table and pos_table (may be null) are bfloat16 rows of n.
// x16 (may be null): the same as bfloat16.  The rows' rotation angles are taken here too, once for all layers.
cudaError_t launch_embed(const void* table, const void* pos_table, const int* ids, const RowMap& rows, float scale, float* x,
                         void* x16, int tokens, int n, const RotTable& rot, cudaStream_t s, uint64_t* launches);
// q | k | v of a stacked projection (row t at proj + t * ld): bias added; q and k divided by the root mean square of the
// WHOLE projection and weighted, where norms are given, then rotated; k and v into the cache, q left in place.
// `also` (heads 0: none): heads of a mixer beside this one in the same rows, rotated in place.
struct QkvShape { int n_head, n_kv, dk, dv; float eps; };
struct RotHeads { float* x; int heads, dim; RotRows rot; };  // heads * dim values at x + t * ld
cudaError_t launch_qkv_store(float* proj, int ld, const float* bias, const float* q_norm, const float* k_norm, const QkvShape& sh, const RotRows& rot,
                             const RotHeads& also, const LayerKv& kv, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches);
cudaError_t launch_rotate_heads(const RotHeads& h, int ld, int tokens, cudaStream_t s, uint64_t* launches);
// One latent per row (n floats at proj + t * ld): normed, weighted, into the cache.  q16 (may be null): the nq floats at
// q + t * ld as bfloat16 rows of nq.
cudaError_t launch_latent_store(const float* proj, int ld, const float* w, int n, float eps, const LayerKv& kv, const RowMap& rows,
                                int tokens, cudaStream_t s, uint64_t* launches);
cudaError_t launch_rows_bf16(const float* x, int64_t ld, int n, void* out16, int tokens, cudaStream_t s, uint64_t* launches);
// Products per head with bfloat16 weights and f32 activations.
// transposed: y[t][h * cols + c] = sum_r W[h * rows + r][c] x[t * x_ld + h * rows + r]     (a query into the latent space)
// plain:      y[t][h * rows + r] = sum_c W[h * rows + r][c] x[t * x_ld + h * cols + c]     (a latent out of it), times
//             sigmoid(gate[t * gate_ld + h]) when gate is set
cudaError_t launch_head_product_t(const void* w, int heads, int rows, int cols, const float* x, int64_t x_ld, float* y, int tokens,
                                  cudaStream_t s, uint64_t* launches);
cudaError_t launch_head_product(const void* w, int heads, int rows, int cols, const float* x, int64_t x_ld, float* y, const float* gate,
                                int64_t gate_ld, int tokens, cudaStream_t s, uint64_t* launches);
cudaError_t launch_head_transpose(const void* w, int heads, int rows, int cols, void* out, cudaStream_t s, uint64_t* launches);
// Attention over the visible keys.  q: row t at q + t * q_ld.  Results go where SpanOut says.
// one_sequence: the rows are one sequence at consecutive positions; with tensor_cores such rows may run as binary16 MMAs.
// A single decode token whose projection the attention kernel takes in itself (null proj: it is in the cache already):
// the row's stacked q | k | v with launch_qkv_store's arguments, or (latent) its latent with the weights in k_norm.
struct NewToken {
  const float *proj = nullptr, *bias = nullptr, *q_norm = nullptr, *k_norm = nullptr;
  float eps = 0.f;
  bool latent = false;
  RotRows rot{};
};
// Row t's results: n_head * dv values from t * ld on, f32 (out) and/or bfloat16 (out16), times `scale` and, with a gate,
// times sigmoid(gate[t * gate_ld + h * dv + i]) or (head_gate) sigmoid(gate[t * gate_ld + h]).
struct SpanOut {
  float* out;
  void* out16;
  int64_t ld;
  const float* gate;
  int64_t gate_ld;
  bool head_gate;
  float scale;
};
size_t span_scratch_floats(const SpanShape& sh, int max_rows);
bool span_supported(const SpanShape& sh);
cudaError_t launch_span_attention(const float* q, int64_t q_ld, const SpanShape& sh, const LayerKv& kv, const RowMap& rows, int t0, int tokens,
                                  const SpanOut& out, float* scratch, bool tensor_cores, bool one_sequence, const NewToken* nt, cudaStream_t s,
                                  uint64_t* launches);
// x[t] += y[t] / rms(y[t]) * w, y given as `slices` partial sums `slice_stride` floats apart; x16 (may be null): the new x
cudaError_t launch_norm_add(float* x, const float* y, int slices, int64_t slice_stride, const float* w, float eps, void* x16, int tokens, int n,
                            cudaStream_t s, uint64_t* launches);
// x[t] += y[t] (slices 0: nothing to add), then, with w, h[t] = x[t] / rms(x[t]) * w as f32 (h) and / or bfloat16 (h16)
cudaError_t launch_add_norm(float* x, const float* y, int slices, int64_t slice_stride, const float* w, float eps, float* h, void* h16, int tokens,
                            int n, cudaStream_t s, uint64_t* launches);
// the gated unit of a stacked product: row t of gu is gate | up, n each
cudaError_t launch_gated_unit(const float* gu, const GluShape& sh, float* out, void* out16, int tokens, cudaStream_t s, uint64_t* launches);

// ---- recurrent mixers (llr_recurrent.cu): a state per sequence instead of cached positions ----
// The groups of a batch: group i has the rows [first[i], first[i + 1]) of one sequence at consecutive positions; null: one
// group of all rows.  A group whose first row stands at position 0 starts from a state of zeros, whatever memory holds.
struct RowGroups {
  const int* first;
  int n, longest;
};
// A mixer's state of sequence q lies at state + q * stride.
struct StateView {
  float* state;
  int64_t stride;
};
// Short causal convolution per channel over the rows of a sequence: w [taps][channels], the last tap weighs the row itself.
// bias is added to the inputs, out_bias to the results (both may be null); tail: the state's last taps - 1 inputs
// [taps - 1][channels].
struct ConvShape {
  const float *w, *bias, *out_bias;
  int channels, taps;
  StateView tail;
};
// What follows a head's result o (vdim values): o / rms(o) (times weight), times sigmoid or silu of its gate row, times
// scale; f32 and / or bfloat16 rows at t * ld.
struct HeadOut {
  const float *weight, *gate;
  int64_t gate_ld;
  bool silu;
  float eps, scale;
  float* out;
  void* out16;
  int64_t ld;
};
// Matrix states S [dim][vdim] per head, one column of S per eight lanes, f32.  Row t: q, k (n_kv heads of dim, head h reads
// h / (n_head / n_kv)) and v (n_head of vdim) at + t * ld.
//   retention (g null):  S = decay[h] S + (k scale) v^T, o = S^T q; a single row may come unrotated (rot)
//   delta rule:          S = diag(g) S, u = beta (v - S^T k), S += k u^T, o = S^T q; g [n_head][dim], beta [n_head],
//                        kq [n_kv] = k . q at + t * ld too
struct MatrixScan {
  const float *q, *k, *v, *g, *beta, *kq, *decay;
  int64_t ld, v_ld;
  int n_head, n_kv, dim, vdim;
  float k_scale;
  RotRows rot;
  StateView state;
  // delta rule: the convolution's inputs, whose last rows replace the state's tail behind the scan
  const float* conv_in;
  int64_t conv_ld;
  ConvShape conv;
};
bool matrix_scan_supported(int dim, int vdim);
// Long groups go by blocks of four rows, from records made of their queries, keys and decays (scan_record_floats of them, 16-byte
// aligned; rows and vectors on 16-byte boundaries).  With `records` the launch takes that form: for retention it makes them, for the
// delta rule launch_delta_prepare has (q, k, g, beta and kq are not read then).
bool scan_by_blocks(int dim, int vdim, const RowGroups& groups);
size_t scan_record_floats(int n_head, int dim, bool delta, int tokens, int n_seq);
// o_scratch: [tokens][n_head * vdim] floats
cudaError_t launch_matrix_scan(const MatrixScan& m, const HeadOut& out, float* records, const RowGroups& groups, const RowMap& rows, int tokens,
                               float* o_scratch, cudaStream_t s, uint64_t* launches);
// Inputs of the delta rule from a row of projections q | k | v: convolution, silu, q and k as unit vectors (x / sqrt(sum x^2 +
// unit_eps)), q times q_scale; g = exp(-rate[h] softplus(a + step_bias)), beta = sigmoid(b).
// Row t of prep (delta_prep_floats): q | k | v | g | beta | k . q.  With `records`: those, and rows of n_head * vdim values v in prep.
struct DeltaShape {
  int n_head, n_kv, dim, vdim;
  float q_scale, unit_eps;
  const float *rate, *step_bias;  // [n_head], [n_head * dim]
};
int delta_prep_floats(const DeltaShape& d);
cudaError_t launch_delta_prepare(const float* proj, int64_t ld, const float* a, const float* b, const DeltaShape& d, const ConvShape& conv, float* prep,
                                 float* records, const RowGroups& groups, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches);
// u[t] = convolution of the rows at x + t * ld.  u16 (may be null): u as three bfloat16 parts whose sum it is, per block of
// `block` channels: [channels / block][3][block].
cudaError_t launch_conv_rows(const float* x, int64_t ld, const ConvShape& conv, float* u, void* u16, int block, const RowMap& rows, int tokens,
                             cudaStream_t s, uint64_t* launches);
// Real-gated linear recurrence per channel: r, i = sigmoid(gates + gate_bias) (row t of gates: per block r | i), log a =
// -rate r, S = a S + sqrt(1 - a^2) i u; result S gelu(y + y_bias).
struct GatedScan {
  const float *gates, *gate_bias, *u, *rate, *y, *y_bias;
  int64_t y_ld;
  int width, block;
  StateView state;
  const float* conv_in;  // as in MatrixScan
  int64_t conv_ld;
  ConvShape conv;
  float* out;
  void* out16;
  int64_t ld;
  float scale;
};
cudaError_t launch_gated_scan(const GatedScan& g, const RowGroups& groups, const RowMap& rows, int tokens, cudaStream_t s, uint64_t* launches);
// W with every block of `cols` columns three times in a row, for products with u16 (once per session)
cudaError_t launch_triple_columns(const void* w, int64_t rows, int cols, void* out, cudaStream_t s, uint64_t* launches);

// *flag_dev = 1 when the two device byte ranges differ (both 16-byte aligned), else 0
cudaError_t launch_bytes_differ(const void* a, const void* b, size_t n, int* flag_dev, cudaStream_t stream, uint64_t* launches);

// Seeded synthetic packed blocks (see llama_rust_b200/synth.py for the recipe).
cudaError_t launch_synth(int dtype, int64_t rows, int64_t cols, uint64_t seed, uint8_t* w,
                         cudaStream_t stream, uint64_t* launches);

}  // namespace llr
