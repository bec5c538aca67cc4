// Decoders described layer by layer, as sessions (included by llr_exec.cu, inside its unnamed namespace): checks of the
// description, device copies and buffers, and the forward pass over a batch's rows.  The session around it -- sequences,
// paged pool, batches, logits, greedy decode and its graph -- is the one of the Llama walk.

bool bf16_operand(const llr_matrix* m) { return m->dtype == LLR_DTYPE_BF16 && gemm_bf16_supported(m->dev, m->rows, m->cols); }

// bucket(n) for n = 0 .. bias_max; from bias_max on every distance is in the last one.  A value within 1e-9 of a whole
// number is taken for it: the quotient of two logarithms misses an exact power by a rounding.
int distance_bucket(int n, int n_bucket, int bias_max) {
  const int half = n_bucket / 2;
  if (n < half) return n;
  const double v = std::log((double)n / half) / std::log((double)bias_max / half) * (n_bucket - half);
  return (int)std::min<double>(n_bucket - 1, half + std::floor(v + 1e-9));
}

DeltaShape delta_shape(const LayeredDecoder::Mixer& M) {
  const llr_mixer& x = M.mx;
  return DeltaShape{(int)x.n_head, (int)x.n_head_kv, (int)x.dim, (int)x.vdim, x.scale, x.unit_eps, M.decay, M.step_bias};
}

// "" when the mixer is one the session can run; fills the derived sizes
std::string mixer_check(llr_exec* e, const llr_decoder_model* m, size_t li, const llr_mixer& x, const std::vector<LayeredDecoder::Layer>& before,
                        LayeredDecoder::Mixer* out) {
  const size_t H = x.n_head, G = x.n_head_kv;
  auto shape = [&](const llr_matrix* w, size_t rows, size_t cols) {
    return w && w->owner == e && (size_t)w->rows == rows && (size_t)w->cols == cols;
  };
  LayeredDecoder::Mixer& M = *out;
  M.mx = x;
  const bool channels = x.kind == LLR_MIXER_GATED_LINEAR;
  if (!std::isfinite(x.scale)) return "scale is not a number";
  if (!channels && (H == 0 || H > 4096 || x.dim == 0 || x.dim > 1024 || x.vdim == 0 || x.vdim > 1024)) return "heads or head sizes out of range";
  if (x.window > (1u << 30) || x.keep_first > (1u << 30)) return "window out of range";
  if (x.rot_dims > 0 && (x.rot_dims % 2 != 0 || x.rot_dims > x.dim || !x.rot_freq)) return "rot_dims must be even and at most dim";
  if (x.rot_dims > 0 && x.kind != LLR_MIXER_ATTENTION && x.kind != LLR_MIXER_RETENTION) return "this mixer has no rotation";
  if (x.sink && x.kind != LLR_MIXER_ATTENTION) return "only attention has a sink";
  M.out_cols = (int)(H * x.vdim);
  M.q_rows = (int)(H * x.dim);
  if (x.kind == LLR_MIXER_ATTENTION) {
    if (G == 0 || H % G != 0) return "n_head must be a multiple of n_head_kv";
    if (x.gate > LLR_GATE_HEAD) return "unknown gate";
    if (x.kv_from >= 0) return "only latent attention reads another layer's cache";
    if (x.n_bucket > 0 && (!x.rel || x.n_bucket < 2 || x.bias_max <= x.n_bucket / 2 || x.bias_max > (1u << 24))) return "distance bias out of range";
    M.gate_col = (int)(H * x.dim + G * x.dim + G * x.vdim);
    M.in_rows = M.gate_col + (int)(x.gate == LLR_GATE_ELEMENT ? H * x.vdim : x.gate == LLR_GATE_HEAD ? H : 0);
    M.span = SpanShape{(int)H, (int)G, (int)x.dim, (int)x.vdim, (int)x.window, (int)x.keep_first, (int)m->n_ctx, x.scale, nullptr, 0, nullptr};
  } else if (x.kind == LLR_MIXER_LATENT) {
    if (x.kv_rank == 0) return "kv_rank must be positive";
    if (x.gate != LLR_GATE_NONE && x.gate != LLR_GATE_HEAD) return "latent attention takes a head gate or none";
    if (x.n_bucket > 0) return "latent attention has no distance bias";
    if (x.kv_from >= 0) {
      if ((size_t)x.kv_from >= li) return "kv_from must name an earlier layer";
      const llr_mixer& src = before[x.kv_from].mixers[0].mx;
      if (src.kind != LLR_MIXER_LATENT || src.kv_from >= 0 || src.kv_rank != x.kv_rank) return "kv_from must name a latent layer with latents of its own and the same kv_rank";
      M.own_kv = false;
    }
    if (!shape(x.up_k, H * x.dim, x.kv_rank) || !shape(x.up_v, H * x.vdim, x.kv_rank) || x.up_k->dtype != LLR_DTYPE_BF16 || x.up_v->dtype != LLR_DTYPE_BF16)
      return "up_k / up_v must be BF16 matrices of n_head * dim / n_head * vdim rows and kv_rank columns";
    M.gate_col = (int)(H * x.dim + (M.own_kv ? x.kv_rank : 0));
    M.in_rows = M.gate_col + (x.gate == LLR_GATE_HEAD ? (int)H : 0);
    M.span = SpanShape{(int)H, 1, (int)x.kv_rank, (int)x.kv_rank, (int)x.window, (int)x.keep_first, (int)m->n_ctx, x.scale, nullptr, 0, nullptr};
  } else if (x.kind == LLR_MIXER_RETENTION) {
    if (!x.decay || !matrix_scan_supported((int)x.dim, (int)x.vdim)) return "retention needs a decay per head";
    M.gate_col = (int)(2 * H * x.dim + H * x.vdim);
    M.in_rows = M.gate_col + M.out_cols;
    M.recurrent = true;
  } else if (x.kind == LLR_MIXER_DELTA) {
    if (G == 0 || H % G != 0) return "n_head must be a multiple of n_head_kv";
    if (x.taps == 0 || x.taps > 64 || !x.conv || !x.decay || !x.step_bias || !x.head_norm || x.decay_rank == 0 || x.gate_rank == 0 || !(x.unit_eps >= 0.f))
      return "a part of the delta rule is missing";
    if (!shape(x.decay_up, H * x.dim, x.decay_rank) || !shape(x.gate_up, H * x.vdim, x.gate_rank) || x.decay_up->dtype != LLR_DTYPE_BF16 || x.gate_up->dtype != LLR_DTYPE_BF16)
      return "decay_up / gate_up must be BF16 matrices of n_head * dim / n_head * vdim rows";
    if (!matrix_scan_supported((int)x.dim, (int)x.vdim)) return "head sizes outside the scan kernels";
    M.channels = (int)(2 * G * x.dim + H * x.vdim);
    M.gate_col = M.channels;  // the low-rank rows: decay, gate; beta behind them
    M.in_rows = M.channels + (int)(x.decay_rank + x.gate_rank + H);
    M.recurrent = true;
  } else if (channels) {
    if (x.width == 0 || x.width > (1u << 20) || x.blocks == 0 || x.width % x.blocks != 0) return "width must be a multiple of blocks";
    if (x.taps == 0 || x.taps > 64 || !x.conv || !x.conv_bias || !x.decay || !x.gate_bias) return "a part of the gated recurrence is missing";
    if (!shape(x.gates, 2 * (size_t)x.width, x.width / x.blocks) || x.gates->dtype != LLR_DTYPE_BF16) return "gates must be a BF16 matrix of 2 width rows";
    M.channels = (int)x.width;
    M.out_cols = (int)x.width;
    M.in_rows = 2 * (int)x.width;
    M.recurrent = true;
  } else {
    return "unknown mixer";
  }
  if (!M.recurrent && !span_supported(M.span)) return "head sizes, latent size or context length outside the attention kernels";
  return "";
}

// "" when the layer is one the session can run; fills its mixers and what it shares between them
std::string layered_check(llr_exec* e, const llr_decoder_model* m, size_t li, const std::vector<LayeredDecoder::Layer>& before, LayeredDecoder::Layer* out) {
  const llr_decoder_layer& D = m->layers[li];
  const size_t E = m->n_embd;
  auto shape = [&](const llr_matrix* w, size_t rows, size_t cols) {
    return w && w->owner == e && (size_t)w->rows == rows && (size_t)w->cols == cols;
  };
  LayeredDecoder::Layer& L = *out;
  L.mlp = D.mlp;
  L.in_proj = D.mixer.in_proj;
  L.out_proj = D.mixer.out_proj;
  L.mixers.resize(D.beside ? 2 : 1);
  std::string why = mixer_check(e, m, li, D.mixer, before, &L.mixers[0]);
  if (!why.empty()) return why;
  size_t rows = L.mixers[0].in_rows, cols = L.mixers[0].out_cols;
  if (D.beside) {
    LayeredDecoder::Mixer& M = L.mixers[1];
    if (D.mixer.kind == LLR_MIXER_LATENT || D.beside->kind == LLR_MIXER_LATENT) return "latent attention stands alone in its layer";
    if (D.beside->in_proj || D.beside->out_proj) return "a mixer beside another has no matrices in_proj / out_proj of its own";
    why = mixer_check(e, m, li, *D.beside, before, &M);
    if (!why.empty()) return "beside: " + why;
    if (!std::isfinite(D.mixer_scale) || !std::isfinite(D.beside_scale)) return "scale is not a number";
    L.mixers[0].scale = D.mixer_scale;
    M.scale = D.beside_scale;
    M.in_col = (int)((rows + 7) & ~(size_t)7);
    M.out_col = (int)cols;
    rows = M.in_col + M.in_rows;
    cols += M.out_cols;
  }
  const llr_matrix* in = L.in_proj;
  if (!in || in->owner != e || (size_t)in->cols != E || (size_t)in->rows < rows || !shape(L.out_proj, E, cols)) return "in_proj / out_proj do not match the mixer's sizes";
  if (!D.mixer_norm || (D.mlp.n_ff > 0 && !D.mlp_norm)) return "a norm is missing";
  if (D.mlp.unit > LLR_UNIT_GELU) return "unknown gated unit";
  if (D.mlp.n_ff > 0 && (!shape(D.mlp.gate_up, 2 * (size_t)D.mlp.n_ff, E) || !shape(D.mlp.down, E, D.mlp.n_ff) || (D.mlp.unit == LLR_UNIT_CLAMPED && !(D.mlp.limit >= 0.f))))
    return "gate_up / down do not match n_ff, or the limit is negative";
  return "";
}

// One forward pass over the rows of a batch: what its layers share
struct LayeredPass {
  llr_session* s;
  size_t n;
  RowMap rows;
  RowGroups groups;
  bool tc;  // rows enough for the tensor cores
  llr_exec* e;
  LayeredDecoder& D;
  cudaStream_t st;
  uint64_t* lc;

  // y = W x: on the tensor cores from 16-bit rows where the matrix allows (its K range in `slices` partial sums, when the
  // reader adds them), else through the executor's product kernels from f32 rows
  cudaError_t product(const llr_matrix* w, bool on_tc, const float* x, const void* x16, float* y, int* slices) {
    if (!on_tc) {
      if (slices) *slices = 1;
      return session_matmul(e, w, n, x, y);
    }
    Bf16Product p{};
    p.w = w->dev; p.x16 = x16; p.x_ld = p.x_cols = w->cols; p.y = y; p.y_ld = w->rows;
    p.tokens = (int)n; p.rows = (int)w->rows; p.cols = (int)w->cols; p.batch = 1;
    p.slices = slices ? gemm_bf16_slices((int)n, p.rows, p.cols) : 1;
    p.slice_stride = (int64_t)n * w->rows;
    if (slices) *slices = p.slices;
    return launch_gemm_bf16(p, st, e->err_flag, lc);
  }

  RotRows rotation(const LayeredDecoder::Mixer& M) const { return RotRows{D.angles + M.rot_off, (int)D.freq.size(), (int)M.mx.rot_dims}; }
  StateView state(int64_t off) const { return StateView{D.state + off, (int64_t)D.state_floats}; }
  ConvShape convolution(const LayeredDecoder::Mixer& M, const float* bias) const {
    return ConvShape{M.conv, bias, M.conv_bias, M.channels, (int)M.mx.taps, state(M.tail_off)};
  }

  // (a) attention and latent attention: the projection in D.proj becomes result rows in D.att or `h16`
  // `beside` runs once the rows' projections are in place, before the attention itself
  cudaError_t attention(const LayeredDecoder::Layer& L, const LayeredDecoder::Mixer& M, bool out_tc, const void** h16, const std::function<cudaError_t()>& beside) {
    const llr_mixer& mx = M.mx;
    const int N = (int)n;
    const int64_t ld = L.in_proj->rows;
    const bool latent = mx.kind == LLR_MIXER_LATENT, up_tc = tc && M.tc_up;
    const LayerKv kv{s->cache_k + M.k_off, s->cache_k + M.v_off, s->table_dev, (int)s->block_tokens, (int)s->max_blocks, (int64_t)D.block_floats,
                     (int64_t)D.block_floats};
    float* proj = D.proj + M.in_col;
    const float* gate = mx.gate != LLR_GATE_NONE ? proj + M.gate_col : nullptr;
    const float* q = proj;
    int64_t q_ld = ld;
    cudaError_t ce;
    if (latent) {
      if (n > 1 && M.own_kv && (ce = launch_latent_store(proj + M.q_rows, (int)ld, M.kv_norm, (int)mx.kv_rank, D.eps, kv, rows, N, st, lc)) != cudaSuccess) return ce;
      // queries into the latent space, head by head
      if (up_tc) {
        if ((ce = launch_rows_bf16(proj, ld, M.q_rows, D.a16, N, st, lc)) != cudaSuccess) return ce;
        Bf16Product p{};
        p.w = M.up_k_t; p.x16 = D.a16; p.x_ld = p.x_cols = M.q_rows; p.y = D.lat_q; p.y_ld = (int64_t)mx.n_head * mx.kv_rank;
        p.tokens = N; p.rows = (int)mx.kv_rank; p.cols = (int)mx.dim; p.batch = (int)mx.n_head; p.xk = (int)mx.dim; p.slices = 1;
        ce = launch_gemm_bf16(p, st, e->err_flag, lc);
      } else {
        ce = launch_head_product_t(mx.up_k->dev, (int)mx.n_head, (int)mx.dim, (int)mx.kv_rank, proj, ld, D.lat_q, N, st, lc);
      }
      if (ce != cudaSuccess) return ce;
      q = D.lat_q;
      q_ld = (int64_t)mx.n_head * mx.kv_rank;
    } else if (n > 1) {
      const QkvShape sh{(int)mx.n_head, (int)mx.n_head_kv, (int)mx.dim, (int)mx.vdim, D.eps};
      RotHeads also{};
      for (const LayeredDecoder::Mixer& B : L.mixers)  // a retention beside: its queries and keys in the same launch
        if (B.mx.kind == LLR_MIXER_RETENTION && B.mx.rot_dims > 0) also = RotHeads{D.proj + B.in_col, 2 * (int)B.mx.n_head, (int)B.mx.dim, rotation(B)};
      if ((ce = launch_qkv_store(proj, (int)ld, M.in_bias, M.q_norm, M.k_norm, sh, rotation(M), also, kv, rows, N, st, lc)) != cudaSuccess) return ce;
    }
    if ((ce = beside()) != cudaSuccess) return ce;
    // 16-bit result rows where the product that follows takes them: the latent results (lat_o / a16), the heads (att / a16)
    const bool o16 = latent ? up_tc : out_tc;
    SpanOut so{};
    so.ld = latent ? (int64_t)mx.n_head * mx.kv_rank : L.out_proj->cols;
    so.scale = M.scale;
    if (o16) so.out16 = (char*)D.a16 + 2 * (size_t)M.out_col;
    else so.out = latent ? D.lat_o : D.att + M.out_col;
    if (!latent) {
      so.gate = gate;
      so.gate_ld = ld;
      so.head_gate = mx.gate == LLR_GATE_HEAD;
    }
    NewToken nt;  // a single token: the attention kernel norms, rotates and stores it
    nt.eps = D.eps;
    nt.latent = latent;
    if (n == 1 && M.own_kv) nt.proj = latent ? proj + M.q_rows : proj;
    nt.bias = M.in_bias;
    nt.q_norm = M.q_norm;
    nt.k_norm = latent ? M.kv_norm : M.k_norm;
    nt.rot = rotation(M);
    auto attend = [&](size_t t0, size_t len, bool one) {
      return launch_span_attention(q, q_ld, M.span, kv, rows, (int)t0, (int)len, so, D.scratch, tc && len >= (size_t)BF16_TC_MIN_TOKENS, one, &nt, st, lc);
    };
    ce = cudaSuccess;
    if (!rows.row_seq) {
      ce = attend(0, n, true);
    } else {  // a ragged batch: groups long enough for the tensor cores on their own, the runs of shorter ones together
      size_t run = 0, at = 0;
      for (const auto& g : s->batch_groups) {
        if (ce == cudaSuccess && tc && g.second >= (size_t)BF16_TC_MIN_TOKENS) {
          if (g.first > run) ce = attend(run, g.first - run, false);
          if (ce == cudaSuccess) ce = attend(g.first, g.second, true);
          run = g.first + g.second;
        }
        at = g.first + g.second;
      }
      if (ce == cudaSuccess && at > run) ce = attend(run, at - run, false);
    }
    if (ce != cudaSuccess || !latent) return ce;
    // results out of the latent space, times the head gate
    if (up_tc) {
      Bf16Product p{};
      p.w = mx.up_v->dev; p.x16 = D.a16; p.x_ld = p.x_cols = (int64_t)mx.n_head * mx.kv_rank;
      p.y = out_tc ? nullptr : D.att; p.y16 = out_tc ? D.b16 : nullptr; p.y_ld = (int64_t)mx.n_head * mx.vdim;
      p.gate = gate; p.gate_ld = ld;
      p.tokens = N; p.rows = (int)mx.vdim; p.cols = (int)mx.kv_rank; p.batch = (int)mx.n_head; p.xk = (int)mx.kv_rank; p.slices = 1;
      *h16 = D.b16;
      return launch_gemm_bf16(p, st, e->err_flag, lc);
    }
    ce = launch_head_product(mx.up_v->dev, (int)mx.n_head, (int)mx.vdim, (int)mx.kv_rank, D.lat_o, (int64_t)mx.n_head * mx.kv_rank, D.att, gate, ld, N, st, lc);
    if (ce == cudaSuccess && out_tc) ce = launch_rows_bf16(D.att, (int64_t)mx.n_head * mx.vdim, (int)(mx.n_head * mx.vdim), D.a16, N, st, lc);
    return ce;
  }

  HeadOut head_out(const LayeredDecoder::Layer& L, const LayeredDecoder::Mixer& M, bool out_tc) const {
    HeadOut o{};
    o.weight = M.head_norm;
    o.eps = D.eps;
    o.scale = M.scale;
    o.ld = L.out_proj->cols;
    if (out_tc) o.out16 = (char*)D.a16 + 2 * (size_t)M.out_col;
    else o.out = D.att + M.out_col;
    return o;
  }

  // (b) retention
  cudaError_t retention(const LayeredDecoder::Layer& L, const LayeredDecoder::Mixer& M, bool out_tc) {
    const llr_mixer& mx = M.mx;
    const int64_t ld = L.in_proj->rows;
    float* proj = D.proj + M.in_col;
    const int nq = (int)(mx.n_head * mx.dim);
    if (n > 1 && mx.rot_dims > 0) {  // a single row is rotated by the scan; beside attention the store kernel has done it
      bool done = false;
      for (const LayeredDecoder::Mixer& B : L.mixers) done = done || B.mx.kind == LLR_MIXER_ATTENTION;
      cudaError_t ce;
      if (!done && (ce = launch_rotate_heads(RotHeads{proj, 2 * (int)mx.n_head, (int)mx.dim, rotation(M)}, (int)ld, (int)n, st, lc)) != cudaSuccess) return ce;
    }
    MatrixScan m{};
    m.q = proj; m.k = proj + nq; m.v = proj + 2 * nq;
    m.decay = M.decay;
    m.ld = m.v_ld = ld;
    m.n_head = m.n_kv = (int)mx.n_head; m.dim = (int)mx.dim; m.vdim = (int)mx.vdim;
    m.k_scale = mx.scale;
    if (n == 1) m.rot = rotation(M);
    m.state = state(M.state_off);
    HeadOut o = head_out(L, M, out_tc);
    o.gate = proj + M.gate_col;
    o.gate_ld = ld;
    o.silu = true;
    const bool blocks = scan_by_blocks(m.dim, m.vdim, groups) && ld % 4 == 0 && (((uintptr_t)m.q | (uintptr_t)m.k) & 15) == 0;
    return launch_matrix_scan(m, o, blocks ? D.records : nullptr, groups, rows, (int)n, D.low, st, lc);
  }

  // (c) gated delta rule
  cudaError_t delta_rule(const LayeredDecoder::Layer& L, const LayeredDecoder::Mixer& M, bool out_tc) {
    const llr_mixer& mx = M.mx;
    const int64_t ld = L.in_proj->rows;
    const int N = (int)n, H = (int)mx.n_head, ra = (int)mx.decay_rank, rg = (int)mx.gate_rank, ng = H * (int)mx.dim, nv = H * (int)mx.vdim, nq = (int)(mx.n_head_kv * mx.dim);
    const float* proj = D.proj + M.in_col;
    const float* rank = proj + M.gate_col;
    auto up4 = [](size_t v) { return (v + 3) & ~(size_t)3; };
    float *a = D.low, *gate = a + up4(n * ng), *o_raw = gate + up4(n * nv);
    cudaError_t ce;
    if (tc && M.tc_up) {
      if ((ce = launch_rows_bf16(rank, ld, ra + rg, D.b16, N, st, lc)) != cudaSuccess) return ce;
      Bf16Product p{};
      p.w = mx.decay_up->dev; p.x16 = D.b16; p.x_ld = ra + rg; p.x_cols = ra; p.y = a; p.y_ld = ng;
      p.tokens = N; p.rows = ng; p.cols = ra; p.batch = 1; p.slices = 1;
      if ((ce = launch_gemm_bf16(p, st, e->err_flag, lc)) != cudaSuccess) return ce;
      p.w = mx.gate_up->dev; p.x16 = (const char*)D.b16 + 2 * (size_t)ra; p.x_cols = rg; p.y = gate; p.y_ld = nv;
      p.rows = nv; p.cols = rg;
      if ((ce = launch_gemm_bf16(p, st, e->err_flag, lc)) != cudaSuccess) return ce;
    } else if ((ce = launch_head_product(mx.decay_up->dev, 1, ng, ra, rank, ld, a, nullptr, 0, N, st, lc)) != cudaSuccess ||
               (ce = launch_head_product(mx.gate_up->dev, 1, nv, rg, rank + ra, ld, gate, nullptr, 0, N, st, lc)) != cudaSuccess) {
      return ce;
    }
    const DeltaShape d = delta_shape(M);
    const ConvShape conv = convolution(M, nullptr);
    const bool blocks = scan_by_blocks(d.dim, d.vdim, groups) && ld % 4 == 0 && ((uintptr_t)proj & 15) == 0;
    float* records = blocks ? D.records : nullptr;
    if ((ce = launch_delta_prepare(proj, ld, a, rank + ra + rg, d, conv, D.prep, records, groups, rows, N, st, lc)) != cudaSuccess) return ce;
    MatrixScan m{};
    if (blocks) {
      m.v = D.prep;
      m.v_ld = nv;
    } else {
      m.q = D.prep; m.k = D.prep + nq; m.v = D.prep + 2 * nq; m.g = m.v + nv; m.beta = m.g + ng; m.kq = m.beta + H;
      m.ld = m.v_ld = delta_prep_floats(d);
    }
    m.n_head = H; m.n_kv = (int)mx.n_head_kv; m.dim = (int)mx.dim; m.vdim = (int)mx.vdim;
    m.state = state(M.state_off);
    m.conv_in = proj; m.conv_ld = ld; m.conv = conv;
    HeadOut o = head_out(L, M, out_tc);
    o.gate = gate;
    o.gate_ld = nv;
    return launch_matrix_scan(m, o, records, groups, rows, N, o_raw, st, lc);
  }

  // (d) gated linear recurrence
  cudaError_t gated_linear(const LayeredDecoder::Layer& L, const LayeredDecoder::Mixer& M, bool out_tc) {
    const llr_mixer& mx = M.mx;
    const int64_t ld = L.in_proj->rows;
    const int N = (int)n, W = (int)mx.width, bs = W / (int)mx.blocks;
    const float* proj = D.proj + M.in_col;
    const ConvShape conv = convolution(M, M.in_bias ? M.in_bias + W : nullptr);
    float *u = D.prep, *gates = D.low;
    const bool up_tc = tc && M.tc_up;
    cudaError_t ce;
    if ((ce = launch_conv_rows(proj + W, ld, conv, u, up_tc ? D.b16 : nullptr, bs, rows, N, st, lc)) != cudaSuccess) return ce;
    if (up_tc) {  // u in three parts against the columns three times: 32-bit products
      Bf16Product p{};
      p.w = M.gates3; p.x16 = D.b16; p.x_ld = p.x_cols = 3 * W; p.y = gates; p.y_ld = 2 * W;
      p.tokens = N; p.rows = 2 * bs; p.cols = 3 * bs; p.batch = (int)mx.blocks; p.xk = 3 * bs; p.slices = 1;
      ce = launch_gemm_bf16(p, st, e->err_flag, lc);
    } else {
      ce = launch_head_product(mx.gates->dev, (int)mx.blocks, 2 * bs, bs, u, W, gates, nullptr, 0, N, st, lc);
    }
    if (ce != cudaSuccess) return ce;
    GatedScan g{};
    g.gates = gates; g.gate_bias = M.gate_bias; g.u = u; g.rate = M.decay;
    g.y = proj; g.y_bias = M.in_bias; g.y_ld = ld;
    g.width = W; g.block = bs;
    g.state = state(M.state_off);
    g.conv_in = proj + W; g.conv_ld = ld; g.conv = conv;
    const HeadOut o = head_out(L, M, out_tc);
    g.out = o.out; g.out16 = o.out16; g.ld = o.ld; g.scale = o.scale;
    return launch_gated_scan(g, groups, rows, N, st, lc);
  }

  cudaError_t mixer(const LayeredDecoder::Layer& L, const LayeredDecoder::Mixer& M, bool out_tc, const void** h16, const std::function<cudaError_t()>& beside) {
    if (M.mx.kind == LLR_MIXER_RETENTION) return retention(L, M, out_tc);
    if (M.mx.kind == LLR_MIXER_DELTA) return delta_rule(L, M, out_tc);
    if (M.mx.kind == LLR_MIXER_GATED_LINEAR) return gated_linear(L, M, out_tc);
    return attention(L, M, out_tc, h16, beside);
  }

  cudaError_t feed_forward(const LayeredDecoder::Layer& L, const float* h, int* slices) {
    const int N = (int)n, E = (int)s->cfg.n_embd;
    const GluShape glu{(int)L.mlp.n_ff, L.mlp.limit, L.mlp.alpha, L.mlp.shift, (int)L.mlp.unit};
    const bool down_tc = tc && L.tc_down;
    const MatView gu = view_of(L.mlp.gate_up);
    cudaError_t ce;
    if (tc && L.tc_gu) {  // the gated unit in the product's epilogue
      Bf16Product p{};
      p.w = gu.w; p.x16 = D.x16; p.x_ld = p.x_cols = E; p.y = down_tc ? nullptr : D.act; p.y16 = down_tc ? D.a16 : nullptr; p.y_ld = glu.n;
      p.tokens = N; p.rows = glu.n; p.cols = E; p.batch = 1; p.slices = 1; p.glu = &glu;
      ce = launch_gemm_bf16(p, st, e->err_flag, lc);
    } else if (e->path == PATH_AUTO && n <= 8 && !down_tc && gemv_rows_supported(gu)) {
      ce = launch_gemv_rows_glu(gu, h, D.act, glu, N, st, e->sm_count, lc);
    } else if ((ce = product(L.mlp.gate_up, false, h, nullptr, D.gu, nullptr)) == cudaSuccess) {
      ce = launch_gated_unit(D.gu, glu, down_tc ? nullptr : D.act, down_tc ? D.a16 : nullptr, N, st, lc);
    }
    return ce != cudaSuccess ? ce : product(L.mlp.down, down_tc, D.act, D.a16, D.y, slices);
  }

  cudaError_t run(const int* ids_dev) {
    const int E = (int)s->cfg.n_embd, N = (int)n;
    cudaError_t ce;
    void* x16 = tc ? D.x16 : nullptr;
    if ((ce = launch_embed(D.token_embd->dev, D.pos_embd ? D.pos_embd->dev : nullptr, ids_dev, rows, D.embd_scale, s->x, D.norm_input ? nullptr : x16, N, E,
                           RotTable{D.freq_dev, D.angles, (int)D.freq.size()}, st, lc)) != cudaSuccess)
      return ce;
    int slices = 0;  // of the sublayer result in D.y that the residual stream still lacks (norm_input)
    // what a sublayer reads: the residual stream itself, or its norm
    const float* h = D.norm_input ? s->xn : s->x;
    auto before = [&](const float* w, bool all_tc) {
      return D.norm_input ? launch_add_norm(s->x, D.y, slices, (int64_t)n * E, w, D.eps, tc && all_tc ? nullptr : s->xn, x16, N, E, st, lc) : cudaSuccess;
    };
    auto behind = [&](const float* w) {
      return D.norm_input ? cudaSuccess : launch_norm_add(s->x, D.y, slices, (int64_t)n * E, w, D.eps, x16, N, E, st, lc);
    };
    for (const LayeredDecoder::Layer& L : D.layers) {
      const bool out_tc = tc && L.tc_out;
      if ((ce = before(L.mixer_norm, L.tc_in)) != cudaSuccess || (ce = product(L.in_proj, tc && L.tc_in, h, D.x16, D.proj, nullptr)) != cudaSuccess) return ce;
      const void* h16 = D.a16;
      const std::function<cudaError_t()> nothing = [] { return cudaSuccess; };
      const bool two = L.mixers.size() == 2 && !L.mixers[0].recurrent && L.mixers[1].recurrent && D.side;
      if (two) {  // attention and a recurrence: neither fills the machine, so they run next to each other
        const std::function<cudaError_t()> other = [&] {
          LayeredPass p{s, n, rows, groups, tc, e, D, D.side, lc};
          cudaError_t c;
          if ((c = cudaEventRecord(D.fork, st)) != cudaSuccess || (c = cudaStreamWaitEvent(D.side, D.fork, 0)) != cudaSuccess ||
              (c = p.mixer(L, L.mixers[1], out_tc, &h16, nothing)) != cudaSuccess)
            return c;
          return cudaEventRecord(D.join, D.side);
        };
        if ((ce = mixer(L, L.mixers[0], out_tc, &h16, other)) != cudaSuccess || (ce = cudaStreamWaitEvent(st, D.join, 0)) != cudaSuccess) return ce;
      } else {
        for (const LayeredDecoder::Mixer& M : L.mixers)
          if ((ce = mixer(L, M, out_tc, &h16, nothing)) != cudaSuccess) return ce;
      }
      if ((ce = product(L.out_proj, out_tc, D.att, h16, D.y, &slices)) != cudaSuccess || (ce = behind(L.mixer_norm)) != cudaSuccess) return ce;
      if (L.mlp.n_ff == 0) continue;
      if ((ce = before(L.mlp_norm, L.tc_gu)) != cudaSuccess || (ce = feed_forward(L, h, &slices)) != cudaSuccess || (ce = behind(L.mlp_norm)) != cudaSuccess) return ce;
    }
    return before(nullptr, true);
  }
};

// The layers over n rows (see session_layers): leaves the residual stream in s->x, nothing pending.
cudaError_t layered_layers(llr_session* s, const int* ids_dev, size_t n, const RowMap& rows) {
  llr_exec* e = s->owner;
  RowGroups groups{nullptr, 1, (int)n};
  if (rows.row_seq) {
    groups = RowGroups{s->dec->group_first, (int)s->batch_groups.size(), 0};
    for (const auto& g : s->batch_groups) groups.longest = std::max(groups.longest, (int)g.second);
  }
  const bool tc = (e->path == PATH_AUTO || e->path == PATH_TC) && n >= (size_t)BF16_TC_MIN_TOKENS;
  return LayeredPass{s, n, rows, groups, tc, e, *s->dec, e->stream, &e->ctr.launches}.run(ids_dev);
}

int layered_create(llr_exec* e, const llr_decoder_model* m, size_t n_seq, size_t kv_blocks, size_t block_tokens, llr_session** out) {
  if (!e) return LLR_ERR_INVALID;
  if (!out) return fail(e, LLR_ERR_INVALID, "null output pointer");
  *out = nullptr;
  if (!m || !m->layers || !m->token_embd || !m->output_norm) return fail(e, LLR_ERR_INVALID, "null model");
  if (m->n_layer == 0 || m->n_embd == 0 || m->n_embd > 65535 || m->n_embd % 4 != 0 || m->n_vocab == 0 || m->n_ctx == 0 || m->n_ctx > (1u << 20) || !(m->norm_eps >= 0.f) ||
      !std::isfinite(m->embd_scale) || m->norm_place > LLR_NORM_INPUT)
    return fail(e, LLR_ERR_INVALID, "decoder configuration out of range (n_embd a multiple of 4)");
  if (n_seq == 0 || n_seq > 4096 || block_tokens == 0 || block_tokens > m->n_ctx)
    return fail(e, LLR_ERR_INVALID, "a session holds 1..4096 sequences and KV blocks of 1..n_ctx positions");
  const llr_matrix* output = m->output ? m->output : m->token_embd;
  const size_t E = m->n_embd, V = m->n_vocab;
  auto table = [&](const llr_matrix* w, size_t min_rows, bool exact) {
    return w->owner == e && w->dtype == LLR_DTYPE_BF16 && (size_t)w->cols == E && (exact ? (size_t)w->rows == min_rows : (size_t)w->rows >= min_rows);
  };
  if (!table(m->token_embd, V, true) || output->owner != e || (size_t)output->rows != V || (size_t)output->cols != E)
    return fail(e, LLR_ERR_INVALID, "token_embd (BF16) / output must be n_vocab x n_embd matrices of this executor");
  if (m->pos_embd && !table(m->pos_embd, m->n_ctx, false)) return fail(e, LLR_ERR_INVALID, "pos_embd must be a BF16 matrix of at least n_ctx x n_embd");
  DeviceGuard guard(e->device);
  std::unique_ptr<LayeredDecoder> D(new LayeredDecoder);
  D->layers.resize(m->n_layer);
  D->embd_scale = m->embd_scale;
  D->eps = m->norm_eps;
  D->norm_input = m->norm_place == LLR_NORM_INPUT;
  D->token_embd = m->token_embd;
  D->pos_embd = m->pos_embd;
  size_t in_rows = 1, lat = 0, heads = 1, ff = 0, a16 = 8, b16 = 8, scratch = 1, prep = 0, low = 0, records = 0;
  auto up4 = [](size_t v) { return (v + 3) & ~(size_t)3; };  // vector loads of keys and values
  for (size_t li = 0; li < m->n_layer; ++li) {
    LayeredDecoder::Layer& L = D->layers[li];
    const std::string why = layered_check(e, m, li, D->layers, &L);
    if (!why.empty()) return fail(e, LLR_ERR_INVALID, "layer " + std::to_string(li) + ": " + why);
    L.tc_in = bf16_operand(L.in_proj);
    L.tc_out = bf16_operand(L.out_proj);
    L.tc_gu = L.mlp.n_ff > 0 && bf16_operand(L.mlp.gate_up);
    L.tc_down = L.mlp.n_ff > 0 && bf16_operand(L.mlp.down);
    in_rows = std::max(in_rows, (size_t)L.in_proj->rows);
    heads = std::max(heads, (size_t)L.out_proj->cols);
    a16 = std::max(a16, (size_t)L.out_proj->cols);
    ff = std::max(ff, (size_t)L.mlp.n_ff);
    for (LayeredDecoder::Mixer& M : L.mixers) {
      const llr_mixer& x = M.mx;
      const size_t H = x.n_head, R = x.kv_rank;
      if (x.rot_dims > 0) {  // rotations that layers share are taken once
        const size_t half = x.rot_dims / 2;
        size_t at = 0;
        while (at + half <= D->freq.size() && !std::equal(x.rot_freq, x.rot_freq + half, D->freq.begin() + at)) ++at;
        if (at + half > D->freq.size()) {
          at = D->freq.size();
          D->freq.insert(D->freq.end(), x.rot_freq, x.rot_freq + half);
        }
        M.rot_off = (int)at;
      }
      if (M.recurrent) {
        const bool channels = x.kind == LLR_MIXER_GATED_LINEAR;
        M.state_off = (int64_t)D->state_floats;
        D->state_floats += up4(channels ? x.width : H * x.dim * x.vdim);
        M.tail_off = (int64_t)D->state_floats;
        if (M.channels > 0) D->state_floats += up4((size_t)(x.taps - 1) * M.channels);
        if (!channels) records = std::max(records, scan_record_floats((int)H, (int)x.dim, x.kind == LLR_MIXER_DELTA, (int)std::min<size_t>(512, m->n_ctx * n_seq), (int)n_seq));
        if (x.kind == LLR_MIXER_RETENTION) {
          low = std::max(low, H * x.vdim);
        } else if (x.kind == LLR_MIXER_DELTA) {
          M.tc_up = bf16_operand(x.decay_up) && bf16_operand(x.gate_up);
          low = std::max(low, H * x.dim + 2 * H * x.vdim);
          prep = std::max(prep, (size_t)delta_prep_floats(delta_shape(M)));
          b16 = std::max(b16, (size_t)x.decay_rank + x.gate_rank);
        } else {
          M.tc_up = bf16_operand(x.gates);
          low = std::max(low, 2 * (size_t)x.width);
          prep = std::max(prep, (size_t)x.width);
          b16 = std::max(b16, 3 * (size_t)x.width);
        }
        continue;
      }
      if (!M.own_kv) {
        M.k_off = D->layers[x.kv_from].mixers[0].k_off;
        M.v_off = M.k_off;
      } else {
        M.k_off = (int64_t)D->block_floats;
        D->block_floats += up4((size_t)M.span.n_kv * block_tokens * M.span.dk);
        M.v_off = M.k_off;
        if (x.kind == LLR_MIXER_ATTENTION) {
          M.v_off = (int64_t)D->block_floats;
          D->block_floats += up4((size_t)M.span.n_kv * block_tokens * M.span.dv);
        }
      }
      if (x.kind == LLR_MIXER_LATENT) {
        lat = std::max(lat, H * R);
        M.tc_up = bf16_operand(x.up_v) && x.dim % 8 == 0;
        a16 = std::max(a16, std::max(H * R, (size_t)M.q_rows));
        b16 = std::max(b16, H * x.vdim);
      }
      scratch = std::max(scratch, span_scratch_floats(M.span, 512));
    }
  }
  a16 = std::max(a16, ff);
  llr_session* s = new (std::nothrow) llr_session();
  if (!s) return fail(e, LLR_ERR_OOM, "host allocation failed");
  s->owner = e;
  s->cfg.n_layer = m->n_layer;
  s->cfg.n_embd = m->n_embd;
  s->cfg.n_vocab = m->n_vocab;
  s->cfg.n_ctx = m->n_ctx;
  s->cfg.rms_eps = m->norm_eps;
  s->embd = m->token_embd;
  s->output = output;
  session_pool(s, n_seq, kv_blocks, block_tokens);
  s->logits_rows = std::max(n_seq, std::min<size_t>(s->max_batch, 64));
  const size_t B = s->max_batch;
  cudaError_t ce = cudaSuccess;
  auto alloc = [&](float** p, size_t n) { if (ce == cudaSuccess) ce = cudaMalloc((void**)p, n * sizeof(float)); };
  auto ialloc = [&](int** p, size_t n) { if (ce == cudaSuccess) ce = cudaMalloc((void**)p, n * sizeof(int)); };
  std::vector<float> by_tap;  // weights of a convolution, [taps][channels]
  auto taps_first = [&](const float* w, size_t channels, size_t taps) {
    by_tap.resize(channels * taps);
    for (size_t c = 0; c < channels; ++c)
      for (size_t j = 0; j < taps; ++j) by_tap[j * channels + c] = w[c * taps + j];
    return by_tap.data();
  };
  auto copy = [&](const float* host, size_t n, float** dev) {
    if (!host || n == 0 || ce != cudaSuccess) return;
    ce = cudaMalloc((void**)dev, n * sizeof(float));
    if (ce == cudaSuccess) ce = cudaMemcpy(*dev, host, n * sizeof(float), cudaMemcpyHostToDevice);
  };
  for (size_t li = 0; li < m->n_layer && ce == cudaSuccess; ++li) {
    LayeredDecoder::Layer& L = D->layers[li];
    copy(m->layers[li].mixer_norm, E, &L.mixer_norm);
    copy(m->layers[li].mlp_norm, L.mlp.n_ff > 0 ? E : 0, &L.mlp_norm);
    for (LayeredDecoder::Mixer& M : L.mixers) {
      llr_mixer& x = M.mx;
      const size_t H = x.n_head, G = x.n_head_kv;
      std::vector<float> rate;  // of the decays, whose logarithms are -rate times something positive
      if (x.kind == LLR_MIXER_ATTENTION) {
        copy(x.in_bias, (size_t)M.gate_col, &M.in_bias);
        copy(x.q_norm, H * x.dim, &M.q_norm);
        copy(x.k_norm, G * x.dim, &M.k_norm);
        copy(x.sink, H, &M.sink);
        M.span.sink = M.sink;
        if (x.n_bucket > 0) {  // one value per head and distance: no logarithm in the kernels
          const size_t len = (size_t)std::min<uint64_t>(x.bias_max, m->n_ctx) + 1;
          std::vector<float> by_distance(H * len);
          for (size_t d = 0; d < len; ++d) {
            const int b = distance_bucket((int)d, (int)x.n_bucket, (int)x.bias_max);
            for (size_t h = 0; h < H; ++h) by_distance[h * len + d] = x.rel[(size_t)b * H + h];
          }
          copy(by_distance.data(), by_distance.size(), &M.bias);
          M.span.bias = M.bias;
          M.span.bias_len = (int)len;
        }
      } else if (x.kind == LLR_MIXER_LATENT) {
        if (M.own_kv) copy(x.kv_norm, x.kv_rank, &M.kv_norm);
        if (M.tc_up) {
          if (ce == cudaSuccess) ce = cudaMalloc(&M.up_k_t, (size_t)x.up_k->rows * x.up_k->cols * 2 + 256);
          if (ce == cudaSuccess) ce = launch_head_transpose(x.up_k->dev, (int)H, (int)x.dim, (int)x.kv_rank, M.up_k_t, e->stream, &e->ctr.launches);
        }
      } else if (x.kind == LLR_MIXER_RETENTION) {
        copy(x.decay, H, &M.decay);
      } else if (x.kind == LLR_MIXER_DELTA) {
        for (size_t h = 0; h < H; ++h) rate.push_back((float)std::exp((double)x.decay[h]));
        copy(rate.data(), H, &M.decay);
        copy(taps_first(x.conv, M.channels, x.taps), (size_t)M.channels * x.taps, &M.conv);
        copy(x.step_bias, H * x.dim, &M.step_bias);
        copy(x.head_norm, x.vdim, &M.head_norm);
      } else {
        for (size_t c = 0; c < x.width; ++c) {
          const double z = x.decay[c];
          rate.push_back((float)(x.scale * (z > 0 ? z + std::log1p(std::exp(-z)) : std::log1p(std::exp(z)))));
        }
        copy(rate.data(), x.width, &M.decay);
        copy(taps_first(x.conv, M.channels, x.taps), (size_t)M.channels * x.taps, &M.conv);
        copy(x.conv_bias, x.width, &M.conv_bias);
        copy(x.gate_bias, 2 * (size_t)x.width, &M.gate_bias);
        if (x.in_bias) {
          copy(x.in_bias, 2 * (size_t)x.width, &M.in_bias);
        } else {
          const std::vector<float> zero(2 * (size_t)x.width, 0.f);
          copy(zero.data(), zero.size(), &M.in_bias);
        }
        if (M.tc_up) {
          if (ce == cudaSuccess) ce = cudaMalloc(&M.gates3, (size_t)x.gates->rows * x.gates->cols * 6 + 256);
          if (ce == cudaSuccess) ce = launch_triple_columns(x.gates->dev, x.gates->rows, (int)x.gates->cols, M.gates3, e->stream, &e->ctr.launches);
        }
      }
      // the device copies are the ones used
      x.in_bias = x.q_norm = x.k_norm = x.kv_norm = x.rel = x.sink = x.conv = x.conv_bias = x.gate_bias = x.decay = x.step_bias = x.head_norm = nullptr;
      x.rot_freq = nullptr;
    }
  }
  auto alloc16 = [&](void** p, size_t n) { if (ce == cudaSuccess) ce = cudaMalloc(p, n * 2 + 256); };
  copy(m->output_norm, E, &s->out_norm);
  alloc(&s->x, B * E); alloc(&s->xn, B * E);
  alloc(&s->logits, s->logits_rows * V); alloc(&s->last_x, s->logits_rows * E); alloc(&s->arg_part, 512);
  alloc(&s->cache_k, s->n_blocks * D->block_floats + 64);
  alloc(&D->proj, B * in_rows); alloc(&D->att, B * heads); alloc(&D->scratch, scratch);
  if (lat) { alloc(&D->lat_q, B * lat); alloc(&D->lat_o, B * lat); }
  if (ff) { alloc(&D->gu, B * 2 * ff); alloc(&D->act, B * ff); }
  if (D->state_floats) { alloc(&D->state, n_seq * D->state_floats); alloc(&D->low, B * low + 8); ialloc(&D->group_first, n_seq + 1); }
  if (prep) alloc(&D->prep, B * prep);
  for (const auto& L : D->layers)
    if (L.mixers.size() == 2 && !D->side && ce == cudaSuccess) {
      ce = cudaStreamCreateWithFlags(&D->side, cudaStreamNonBlocking);
      if (ce == cudaSuccess) ce = cudaEventCreateWithFlags(&D->fork, cudaEventDisableTiming);
      if (ce == cudaSuccess) ce = cudaEventCreateWithFlags(&D->join, cudaEventDisableTiming);
    }
  if (records) alloc(&D->records, records);
  if (!D->freq.empty()) {
    if (ce == cudaSuccess) ce = cudaMalloc((void**)&D->freq_dev, D->freq.size() * sizeof(double));
    if (ce == cudaSuccess) ce = cudaMemcpy(D->freq_dev, D->freq.data(), D->freq.size() * sizeof(double), cudaMemcpyHostToDevice);
    if (ce == cudaSuccess) ce = cudaMalloc((void**)&D->angles, B * D->freq.size() * sizeof(float2));
  }
  for (const auto& L : D->layers)
    for (const llr_matrix* w : {L.out_proj, L.mlp.n_ff > 0 ? L.mlp.down : L.out_proj})
      for (size_t n = 1; n <= B; ++n) D->y_rows = std::max(D->y_rows, n * (size_t)gemm_bf16_slices((int)n, (int)w->rows, (int)w->cols));
  alloc(&D->y, D->y_rows * E);
  alloc16(&D->x16, B * E); alloc16(&D->a16, B * a16); alloc16(&D->b16, B * b16);
  ialloc(&s->pos_dev, 1); ialloc(&s->count_dev, 1);
  ialloc(&s->table_dev, n_seq * s->max_blocks); ialloc(&s->row_pos, B); ialloc(&s->row_seq, B); ialloc(&s->last_rows, s->logits_rows);
  if (ce == cudaSuccess) ce = cudaMemset(s->pos_dev, 0, sizeof(int));
  if (ce == cudaSuccess) ce = cudaMemset(s->table_dev, 0, n_seq * s->max_blocks * sizeof(int));
  if (ce == cudaSuccess) ce = cudaStreamSynchronize(e->stream);
  s->dec = std::move(D);
  if (ce != cudaSuccess) {
    session_release(s);
    delete s;
    return fail_cuda(e, ce, "session buffers");
  }
  e->sessions.insert(s);
  *out = s;
  return LLR_OK;
}
