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

// "" when the layer is one the session can run; fills the derived sizes
std::string layered_check(llr_exec* e, const llr_decoder_model* m, size_t li, const std::vector<LayeredDecoder::Layer>& before, LayeredDecoder::Layer* out) {
  const llr_decoder_layer& D = m->layers[li];
  const llr_mixer& x = D.mixer;
  const size_t E = m->n_embd, H = x.n_head;
  auto shape = [&](const llr_matrix* w, size_t rows, size_t cols) {
    return w && w->owner == e && (size_t)w->rows == rows && (size_t)w->cols == cols;
  };
  if (H == 0 || H > 4096 || x.dim == 0 || x.dim > 1024 || x.vdim == 0 || x.vdim > 1024 || !std::isfinite(x.scale)) return "heads or head sizes out of range";
  if (x.window > (1u << 30) || x.keep_first > (1u << 30)) return "window out of range";
  LayeredDecoder::Layer& L = *out;
  L.mx = x;
  L.mlp = D.mlp;
  L.q_rows = (int)(H * x.dim);
  if (x.kind == LLR_MIXER_ATTENTION) {
    const size_t G = x.n_head_kv;
    if (G == 0 || H % G != 0) return "n_head must be a multiple of n_head_kv";
    if (x.gate != LLR_GATE_NONE && x.gate != LLR_GATE_ELEMENT) return "attention takes an element gate or none";
    if (x.kv_from >= 0) return "only latent attention reads another layer's cache";
    if (x.n_bucket > 0 && (!x.rel || x.n_bucket < 2 || x.bias_max <= x.n_bucket / 2 || x.bias_max > (1u << 24))) return "distance bias out of range";
    L.gate_col = (int)(H * x.dim + G * x.dim + G * x.vdim);
    L.in_rows = L.gate_col + (x.gate == LLR_GATE_ELEMENT ? (int)(H * x.vdim) : 0);
    L.span = SpanShape{(int)H, (int)G, (int)x.dim, (int)x.vdim, (int)x.window, (int)x.keep_first, (int)m->n_ctx, x.scale, nullptr, 0};
  } else if (x.kind == LLR_MIXER_LATENT) {
    if (x.kv_rank == 0) return "kv_rank must be positive";
    if (x.gate != LLR_GATE_NONE && x.gate != LLR_GATE_HEAD) return "latent attention takes a head gate or none";
    if (x.n_bucket > 0) return "latent attention has no distance bias";
    if (x.kv_from >= 0) {
      if ((size_t)x.kv_from >= li) return "kv_from must name an earlier layer";
      const llr_mixer& src = before[x.kv_from].mx;
      if (src.kind != LLR_MIXER_LATENT || src.kv_from >= 0 || src.kv_rank != x.kv_rank) return "kv_from must name a latent layer with latents of its own and the same kv_rank";
      L.own_kv = false;
    }
    if (!shape(x.up_k, H * x.dim, x.kv_rank) || !shape(x.up_v, H * x.vdim, x.kv_rank) || x.up_k->dtype != LLR_DTYPE_BF16 || x.up_v->dtype != LLR_DTYPE_BF16)
      return "up_k / up_v must be BF16 matrices of n_head * dim / n_head * vdim rows and kv_rank columns";
    L.gate_col = (int)(H * x.dim + (L.own_kv ? x.kv_rank : 0));
    L.in_rows = L.gate_col + (x.gate == LLR_GATE_HEAD ? (int)H : 0);
    L.span = SpanShape{(int)H, 1, (int)x.kv_rank, (int)x.kv_rank, (int)x.window, (int)x.keep_first, (int)m->n_ctx, x.scale, nullptr, 0};
  } else {
    return "unknown mixer";
  }
  if (!span_supported(L.span)) return "head sizes, latent size or context length outside the attention kernels";
  if (!shape(x.in_proj, (size_t)L.in_rows, E) || !shape(x.out_proj, E, H * x.vdim)) return "in_proj / out_proj do not match the mixer's sizes";
  if (!D.mixer_norm || (D.mlp.n_ff > 0 && !D.mlp_norm)) return "a norm is missing";
  if (D.mlp.n_ff > 0 && (!shape(D.mlp.gate_up, 2 * (size_t)D.mlp.n_ff, E) || !shape(D.mlp.down, E, D.mlp.n_ff) || !(D.mlp.limit >= 0.f)))
    return "gate_up / down do not match n_ff, or the limit is negative";
  return "";
}

// The layers over n rows (see session_layers): leaves the residual stream in s->x, nothing pending.
cudaError_t layered_layers(llr_session* s, const int* ids_dev, size_t n, const RowMap& rows) {
  llr_exec* e = s->owner;
  LayeredDecoder& D = *s->dec;
  const int E = (int)s->cfg.n_embd, N = (int)n;
  cudaStream_t st = e->stream;
  uint64_t* lc = &e->ctr.launches;
  const bool tc = (e->path == PATH_AUTO || e->path == PATH_TC) && n >= (size_t)BF16_TC_MIN_TOKENS;
  cudaError_t ce;
  // y = W x: on the tensor cores from 16-bit rows where the matrix allows (its K range in `slices` partial sums, when
  // the reader adds them), else through the executor's product kernels from f32 rows
  auto product = [&](const llr_matrix* w, bool on_tc, const float* x, const void* x16, float* y, int* slices) -> cudaError_t {
    if (!on_tc) {
      if (slices) *slices = 1;
      return session_matmul(e, w, n, x, y);
    }
    Bf16Product p{};
    p.w = w->dev; p.x16 = x16; p.x_ld = p.x_cols = w->cols; p.y = y; p.y_ld = w->rows;
    p.tokens = N; p.rows = (int)w->rows; p.cols = (int)w->cols; p.batch = 1;
    p.slices = slices ? gemm_bf16_slices(N, p.rows, p.cols) : 1;
    p.slice_stride = (int64_t)n * w->rows;
    if (slices) *slices = p.slices;
    return launch_gemm_bf16(p, st, e->err_flag, lc);
  };
  if ((ce = launch_embed(D.token_embd->dev, D.pos_embd ? D.pos_embd->dev : nullptr, ids_dev, rows, D.embd_scale, s->x, tc ? D.x16 : nullptr, N, E, st, lc)) !=
      cudaSuccess)
    return ce;
  for (size_t li = 0; li < D.layers.size(); ++li) {
    const LayeredDecoder::Layer& L = D.layers[li];
    const llr_mixer& mx = L.mx;
    const bool latent = mx.kind == LLR_MIXER_LATENT, up_tc = tc && L.tc_up, out_tc = tc && L.tc_out;
    const LayerKv kv{s->cache_k + L.k_off, s->cache_k + L.v_off, s->table_dev, (int)s->block_tokens, (int)s->max_blocks, (int64_t)D.block_floats,
                     (int64_t)D.block_floats};
    if ((ce = product(mx.in_proj, tc && L.tc_in, s->x, D.x16, D.proj, nullptr)) != cudaSuccess) return ce;
    const float* gate = mx.gate != LLR_GATE_NONE ? D.proj + L.gate_col : nullptr;
    const float* q = D.proj;
    int64_t q_ld = L.in_rows;
    if (latent) {
      if (n > 1 && L.own_kv && (ce = launch_latent_store(D.proj + L.q_rows, L.in_rows, L.kv_norm, (int)mx.kv_rank, D.eps, kv, rows, N, st, lc)) != cudaSuccess) return ce;
      // queries into the latent space, head by head
      if (up_tc) {
        if ((ce = launch_rows_bf16(D.proj, L.in_rows, L.q_rows, D.a16, N, st, lc)) != cudaSuccess) return ce;
        Bf16Product p{};
        p.w = L.up_k_t; p.x16 = D.a16; p.x_ld = p.x_cols = L.q_rows; p.y = D.lat_q; p.y_ld = (int64_t)mx.n_head * mx.kv_rank;
        p.tokens = N; p.rows = (int)mx.kv_rank; p.cols = (int)mx.dim; p.batch = (int)mx.n_head; p.xk = (int)mx.dim; p.slices = 1;
        ce = launch_gemm_bf16(p, st, e->err_flag, lc);
      } else {
        ce = launch_head_product_t(mx.up_k->dev, (int)mx.n_head, (int)mx.dim, (int)mx.kv_rank, D.proj, L.in_rows, D.lat_q, N, st, lc);
      }
      if (ce != cudaSuccess) return ce;
      q = D.lat_q;
      q_ld = (int64_t)mx.n_head * mx.kv_rank;
    } else if (n > 1) {
      const QkvShape sh{(int)mx.n_head, (int)mx.n_head_kv, (int)mx.dim, (int)mx.vdim, D.eps};
      if ((ce = launch_qkv_store(D.proj, L.in_rows, L.in_bias, L.q_norm, L.k_norm, sh, kv, rows, N, st, lc)) != cudaSuccess) return ce;
    }
    // 16-bit result rows where the product that follows takes them: the latent results (lat_o / a16), the heads (att / a16)
    const bool o16 = latent ? up_tc : out_tc;
    float* o = o16 ? nullptr : latent ? D.lat_o : D.att;
    void* ob = o16 ? D.a16 : nullptr;
    const float* egate = latent ? nullptr : gate;
    NewToken nt;  // a single token: the attention kernel norms and stores it
    nt.eps = D.eps;
    nt.latent = latent;
    if (n == 1 && L.own_kv) nt.proj = latent ? D.proj + L.q_rows : D.proj;
    nt.bias = L.in_bias;
    nt.q_norm = L.q_norm;
    nt.k_norm = latent ? L.kv_norm : L.k_norm;
    auto attend = [&](size_t t0, size_t len, bool one) {
      return launch_span_attention(q, q_ld, L.span, kv, rows, (int)t0, (int)len, o, ob, egate, L.in_rows, D.scratch, tc && len >= (size_t)BF16_TC_MIN_TOKENS, one,
                                   &nt, st, lc);
    };
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
    if (ce != cudaSuccess) return ce;
    const void* h16 = D.a16;
    if (latent) {  // results out of the latent space, times the head gate
      if (up_tc) {
        Bf16Product p{};
        p.w = mx.up_v->dev; p.x16 = D.a16; p.x_ld = p.x_cols = (int64_t)mx.n_head * mx.kv_rank;
        p.y = out_tc ? nullptr : D.att; p.y16 = out_tc ? D.b16 : nullptr; p.y_ld = (int64_t)mx.n_head * mx.vdim;
        p.gate = gate; p.gate_ld = L.in_rows;
        p.tokens = N; p.rows = (int)mx.vdim; p.cols = (int)mx.kv_rank; p.batch = (int)mx.n_head; p.xk = (int)mx.kv_rank; p.slices = 1;
        ce = launch_gemm_bf16(p, st, e->err_flag, lc);
        h16 = D.b16;
      } else {
        ce = launch_head_product(mx.up_v->dev, (int)mx.n_head, (int)mx.vdim, (int)mx.kv_rank, D.lat_o, (int64_t)mx.n_head * mx.kv_rank, D.att, gate, L.in_rows, N,
                                 st, lc);
        if (ce == cudaSuccess && out_tc) ce = launch_rows_bf16(D.att, (int64_t)mx.n_head * mx.vdim, (int)(mx.n_head * mx.vdim), D.a16, N, st, lc);
      }
      if (ce != cudaSuccess) return ce;
    }
    int slices = 1;
    if ((ce = product(mx.out_proj, out_tc, D.att, h16, D.y, &slices)) != cudaSuccess ||
        (ce = launch_norm_add(s->x, D.y, slices, (int64_t)n * E, L.mixer_norm, D.eps, tc ? D.x16 : nullptr, N, E, st, lc)) != cudaSuccess)
      return ce;
    if (L.mlp.n_ff == 0) continue;
    const GluShape glu{(int)L.mlp.n_ff, L.mlp.limit, L.mlp.alpha, L.mlp.shift};
    const bool down_tc = tc && L.tc_down;
    const MatView gu = view_of(L.mlp.gate_up);
    if (tc && L.tc_gu) {  // the gated unit in the product's epilogue
      Bf16Product p{};
      p.w = gu.w; p.x16 = D.x16; p.x_ld = p.x_cols = E; p.y = down_tc ? nullptr : D.act; p.y16 = down_tc ? D.a16 : nullptr; p.y_ld = glu.n;
      p.tokens = N; p.rows = glu.n; p.cols = E; p.batch = 1; p.slices = 1; p.glu = &glu;
      ce = launch_gemm_bf16(p, st, e->err_flag, lc);
    } else if (e->path == PATH_AUTO && n <= 8 && !down_tc && gemv_rows_supported(gu)) {
      ce = launch_gemv_rows_glu(gu, s->x, D.act, glu, N, st, e->sm_count, lc);
    } else if ((ce = product(L.mlp.gate_up, false, s->x, nullptr, D.gu, nullptr)) == cudaSuccess) {
      ce = launch_clamped_glu(D.gu, glu, down_tc ? nullptr : D.act, down_tc ? D.a16 : nullptr, N, st, lc);
    }
    if (ce != cudaSuccess ||
        (ce = product(L.mlp.down, down_tc, D.act, D.a16, D.y, &slices)) != cudaSuccess ||
        (ce = launch_norm_add(s->x, D.y, slices, (int64_t)n * E, L.mlp_norm, D.eps, tc ? D.x16 : nullptr, N, E, st, lc)) != cudaSuccess)
      return ce;
  }
  return cudaSuccess;
}

int layered_create(llr_exec* e, const llr_decoder_model* m, size_t n_seq, size_t kv_blocks, size_t block_tokens, llr_session** out) {
  if (!e) return LLR_ERR_INVALID;
  if (!out) return fail(e, LLR_ERR_INVALID, "null output pointer");
  *out = nullptr;
  if (!m || !m->layers || !m->token_embd || !m->output_norm) return fail(e, LLR_ERR_INVALID, "null model");
  if (m->n_layer == 0 || m->n_embd == 0 || m->n_embd > 65535 || m->n_embd % 4 != 0 || m->n_vocab == 0 || m->n_ctx == 0 || m->n_ctx > (1u << 20) || !(m->norm_eps >= 0.f) ||
      !std::isfinite(m->embd_scale))
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
  D->token_embd = m->token_embd;
  D->pos_embd = m->pos_embd;
  size_t in_rows = 1, lat = 0, heads = 1, ff = 0, a16 = 8, b16 = 8, scratch = 1;
  auto up4 = [](size_t v) { return (v + 3) & ~(size_t)3; };  // vector loads of keys and values
  for (size_t li = 0; li < m->n_layer; ++li) {
    LayeredDecoder::Layer& L = D->layers[li];
    const std::string why = layered_check(e, m, li, D->layers, &L);
    if (!why.empty()) return fail(e, LLR_ERR_INVALID, "layer " + std::to_string(li) + ": " + why);
    const llr_mixer& x = L.mx;
    if (!L.own_kv) {
      L.k_off = D->layers[x.kv_from].k_off;
      L.v_off = L.k_off;
    } else {
      L.k_off = (int64_t)D->block_floats;
      D->block_floats += up4((size_t)L.span.n_kv * block_tokens * L.span.dk);
      L.v_off = L.k_off;
      if (x.kind == LLR_MIXER_ATTENTION) {
        L.v_off = (int64_t)D->block_floats;
        D->block_floats += up4((size_t)L.span.n_kv * block_tokens * L.span.dv);
      }
    }
    L.tc_in = bf16_operand(x.in_proj);
    L.tc_out = bf16_operand(x.out_proj);
    L.tc_gu = L.mlp.n_ff > 0 && bf16_operand(L.mlp.gate_up);
    L.tc_down = L.mlp.n_ff > 0 && bf16_operand(L.mlp.down);
    const size_t H = x.n_head, R = x.kv_rank;
    in_rows = std::max(in_rows, (size_t)L.in_rows);
    heads = std::max(heads, H * x.vdim);
    a16 = std::max(a16, H * x.vdim);
    if (x.kind == LLR_MIXER_LATENT) {
      lat = std::max(lat, H * R);
      L.tc_up = bf16_operand(x.up_v) && x.dim % 8 == 0;
      a16 = std::max(a16, std::max(H * R, (size_t)L.q_rows));
      b16 = std::max(b16, H * x.vdim);
    }
    ff = std::max(ff, (size_t)L.mlp.n_ff);
    scratch = std::max(scratch, span_scratch_floats(L.span, 512));
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
  auto copy = [&](const float* host, size_t n, float** dev) {
    if (!host || ce != cudaSuccess) return;
    ce = cudaMalloc((void**)dev, n * sizeof(float));
    if (ce == cudaSuccess) ce = cudaMemcpy(*dev, host, n * sizeof(float), cudaMemcpyHostToDevice);
  };
  for (size_t li = 0; li < m->n_layer && ce == cudaSuccess; ++li) {
    LayeredDecoder::Layer& L = D->layers[li];
    const llr_mixer& x = L.mx;
    const size_t H = x.n_head, G = x.n_head_kv;
    copy(m->layers[li].mixer_norm, E, &L.mixer_norm);
    copy(m->layers[li].mlp_norm, L.mlp.n_ff > 0 ? E : 0, &L.mlp_norm);
    if (x.kind == LLR_MIXER_ATTENTION) {
      copy(x.in_bias, (size_t)L.gate_col, &L.in_bias);
      copy(x.q_norm, H * x.dim, &L.q_norm);
      copy(x.k_norm, G * x.dim, &L.k_norm);
      if (x.n_bucket > 0) {  // one value per head and distance: no logarithm in the kernels
        const size_t len = (size_t)std::min<uint64_t>(x.bias_max, m->n_ctx) + 1;
        std::vector<float> by_distance(H * len);
        for (size_t d = 0; d < len; ++d) {
          const int b = distance_bucket((int)d, (int)x.n_bucket, (int)x.bias_max);
          for (size_t h = 0; h < H; ++h) by_distance[h * len + d] = x.rel[(size_t)b * H + h];
        }
        copy(by_distance.data(), by_distance.size(), &L.bias);
        L.span.bias = L.bias;
        L.span.bias_len = (int)len;
      }
    } else {
      if (L.own_kv) copy(x.kv_norm, x.kv_rank, &L.kv_norm);
      if (L.tc_up) {
        if (ce == cudaSuccess) ce = cudaMalloc(&L.up_k_t, (size_t)x.up_k->rows * x.up_k->cols * 2 + 256);
        if (ce == cudaSuccess) ce = launch_head_transpose(x.up_k->dev, (int)H, (int)x.dim, (int)x.kv_rank, L.up_k_t, e->stream, &e->ctr.launches);
      }
    }
    L.mx.in_bias = L.mx.q_norm = L.mx.k_norm = L.mx.kv_norm = L.mx.rel = nullptr;  // the device copies are the ones used
  }
  auto alloc16 = [&](void** p, size_t n) { if (ce == cudaSuccess) ce = cudaMalloc(p, n * 2 + 256); };
  copy(m->output_norm, E, &s->out_norm);
  alloc(&s->x, B * E); alloc(&s->xn, B * E);
  alloc(&s->logits, s->logits_rows * V); alloc(&s->last_x, s->logits_rows * E); alloc(&s->arg_part, 512);
  alloc(&s->cache_k, s->n_blocks * D->block_floats + 64);
  alloc(&D->proj, B * in_rows); alloc(&D->att, B * heads); alloc(&D->scratch, scratch);
  if (lat) { alloc(&D->lat_q, B * lat); alloc(&D->lat_o, B * lat); }
  if (ff) { alloc(&D->gu, B * 2 * ff); alloc(&D->act, B * ff); }
  for (const auto& L : D->layers)
    for (const llr_matrix* w : {L.mx.out_proj, L.mlp.n_ff > 0 ? L.mlp.down : L.mx.out_proj})
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
