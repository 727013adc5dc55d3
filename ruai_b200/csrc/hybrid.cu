// A decoder built from a list of layers: every layer has a token mixer of its own kind.  Tensors by name, caches and states
// per run of a layer, activations and the head are here for both kinds of block; cache growth, graph capture, generation and
// sampling are those of model.cu.  Sandwich blocks are in hybrid_sandwich.cu, parallel blocks here:
//
// The mixer (differential attention over a window with kept first positions, a decayed matrix state with a bonus, a gated
// matrix state) has an optional gated feed-forward beside it.  Both read one RMSNorm of the residual stream, the mixer after
// the token shift, and their sum is added to the stream.
//
// A layer is four launches in a single-token step:
//   1. token_mix      norm, token shift, further interpolations (token_mix.cu)
//   2. dense group    every projection of the mixer and gate / up of the feed-forward, activations fused (dense.cu)
//   3. mixer          attention (attn_span.cu) or recurrence (recurrence.cu), output norms and gates fused
//   4. dense          [W_o | W_down] against [mixer output | feed-forward hidden], added to the residual stream: the two
//                     output projections are one weight, side by side along k
// With 16-bit weights the inputs of the matrix products are bf16; everything else (the stream, norms, projections'
// results, scores, decays, states) is f32.  With 32-bit weights everything is f32.
#include "hybrid_impl.cuh"

#include <algorithm>
#include <cstring>

#include "decode_ops.cuh"

namespace {

constexpr uint64_t kTensorBase = 0x60000000ull;
const char* const kMuNames[MU_N] = {"r", "k", "v", "g", "w"};

void free_lin(Lin& l) {
  if (l.w) ruai_qweight_free(l.w);
  l.w = nullptr;
}

uint64_t id_of(const ruai_model* m, const std::string& name) {
  const HybridTensor* t = hybrid_tensor_by_name(m, name.c_str());
  return t ? t->id : ~0ull;
}
}  // namespace

int hybrid_take(ruai_model* m, const std::string& name, const float** out) {
  DevBuf* b = nullptr;
  if (staged_get(m, id_of(m, name), &b) != RUAI_OK) return model_fail(m, RUAI_ERR_ARG, "tensor '%s' was not set", name.c_str());
  *out = b->as<float>();
  return RUAI_OK;
}
int hybrid_drop(ruai_model* m, const std::string& name) {
  staged_drop(m, id_of(m, name));
  return RUAI_OK;
}
// A vector (or number) moves from the staging map into the model.
int hybrid_move_vec(ruai_model* m, const std::string& name, DevBuf* dst) {
  const float* p;
  RUAI_TRY(hybrid_take(m, name, &p));
  auto it = m->staged.find(id_of(m, name));
  dst->release();
  *dst = it->second;
  m->staged.erase(it);
  return RUAI_OK;
}
int hybrid_build_dense(ruai_model* m, Lin* out, uint32_t n, uint32_t k, uint32_t bits, const std::vector<RowPart>& parts) {
  free_lin(*out);
  RUAI_TRY(ruai_dense_alloc(m->ctx, n, k, bits, &out->w));
  for (const RowPart& p : parts) {
    const float* src;
    RUAI_TRY(hybrid_take(m, p.name, &src));
    const HybridTensor* t = hybrid_tensor_by_name(m, p.name.c_str());
    RUAI_TRY(ruai_dense_put(m->ctx, out->w, src + (size_t)p.src0 * t->cols, p.rows ? p.rows : (uint32_t)t->rows, (uint32_t)t->cols, p.row0, p.row_step, p.col0));
  }
  RUAI_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
  for (const RowPart& p : parts) staged_drop(m, id_of(m, p.name));
  return RUAI_OK;
}

namespace {

SpanParams span_params(const ruai_model* m, uint32_t l, uint32_t B, uint32_t T) {
  const MixLayer& y = m->hy->layers[l];
  const ruai_layer_config& f = y.cfg;
  SpanParams p;
  p.ld = y.qkv_ld();
  p.k_off = 2 * f.heads * f.dim;
  p.v_off = p.k_off + 2 * f.kv_heads * f.dim;
  p.q_norm = y.q_norm.as<float>(); p.k_norm = y.k_norm.as<float>();
  p.eps = m->eps;
  p.T = T; p.G = f.kv_heads; p.rep = f.heads / f.kv_heads; p.maps = 2; p.kd = f.dim; p.vd = f.vdim; p.kdp = y.kdp(); p.vdp = y.vdp();
  p.cap = m->cap; p.window = f.window; p.keep = f.keep_first; p.scale = f.scale;
  p.kcache = m->layers[l].kc.as<float>(); p.vcache = m->layers[l].vc.as<float>();
  p.len = m->d_len.as<int32_t>();
  p.lambda = y.lambda.as<float>();
  p.out_scale = 1.0f - f.diff;
  p.status = m->ctx->status;
  return p;
}

// The projections of layer l and gate / up of its feed-forward, one launch.
int issue_projections(ruai_model* m, uint32_t l, uint32_t m_rows, uint32_t T) {
  Hybrid* y = m->hy;
  MixLayer& L = y->layers[l];
  const ruai_layer_config& f = L.cfg;
  const uint32_t hk = hy_up4(f.heads * f.dim), hv = hy_up4(f.heads * f.vdim);
  float* proj = y->proj.as<float>();
  DenseCall calls[kDenseGroupMax];
  int n = 0;
  auto add = [&](const Lin& w, const DevBuf& x, void* out, uint32_t ld, int act, int dtype) -> DenseCall& {
    DenseCall& d = calls[n++];
    d.w = w.w; d.x = x.p; d.x_ld = y->ldd; d.out = out;
    d.epi.act = act; d.epi.out_dtype = dtype; d.epi.out_ld = ld;
    return d;
  };
  if (L.diff()) {
    add(L.proj[0], y->mix[0], proj, L.qkv_ld(), ACT_NONE, RUAI_F32);
  } else if (f.mixer == RUAI_MIX_WKV) {
    for (int i = 0; i < 4; ++i) add(L.proj[i], y->mix[i], proj + (size_t)i * m_rows * hk, hk, i == MU_G ? ACT_SILU : ACT_NONE, RUAI_F32);
    add(L.proj[MU_W], y->mix[MU_W], y->low.p, y->ldlow, ACT_TANH, y->act);
  } else {
    add(L.proj[0], y->mix[0], proj, hk, ACT_SILU, RUAI_F32);
    DenseCall& d = add(L.proj[1], y->mix[0], proj + (size_t)m_rows * hk, hk, ACT_FORGET, RUAI_F32);
    d.epi.bias = L.f_bias.as<float>(); d.epi.aux = L.lower.as<float>();
    add(L.proj[2], y->mix[0], proj + 2 * (size_t)m_rows * hk, hv, ACT_NONE, RUAI_F32);
  }
  if (f.ff) add(L.up, y->h, (unsigned char*)y->cat.p + (size_t)L.mix_width() * hy_act_bytes(y), y->ldcat, ACT_GEGLU, y->act);
  RUAI_TRY(ruai_dense_launch(m->ctx, calls, n, y->act, m_rows));
  if (f.mixer == RUAI_MIX_WKV && T > 1) {  // the decays; a single-token step works them out in the recurrence kernel
    DenseCall d;
    d.w = L.w2.w; d.x = y->low.p; d.x_ld = y->ldlow; d.out = proj + 4 * (size_t)m_rows * hk;
    d.epi.act = ACT_DECAY; d.epi.bias = L.w0.as<float>(); d.epi.out_ld = hk;
    RUAI_TRY(ruai_dense_launch(m->ctx, &d, 1, y->act, m_rows));
  }
  return RUAI_OK;
}

int issue_output(ruai_model* m, uint32_t l, uint32_t m_rows, float* x) {
  Hybrid* y = m->hy;
  DenseCall d;
  d.w = y->layers[l].od.w; d.x = y->cat.p; d.x_ld = y->ldcat; d.out = x;
  d.epi.resid = x; d.epi.out_ld = m->d;
  return ruai_dense_launch(m->ctx, &d, 1, y->act, m_rows);
}

}  // namespace

int hybrid_issue_head(ruai_model* m, uint32_t out_rows, bool pick, uint32_t len_add) {
  Hybrid* y = m->hy;
  DenseCall d;
  d.w = m->head.w; d.x = y->hx.p; d.x_ld = y->ldd; d.out = m->logits.p;
  if (pick) {
    d.epi.argmax_out = m->d_ids.as<int32_t>(); d.epi.argmax_slots = y->arg_slots.as<int2>();
    d.epi.len_ptr = m->d_len.as<int32_t>(); d.epi.len_add = (int32_t)len_add;
  }
  return ruai_dense_launch(m->ctx, &d, 1, y->act, out_rows);
}

const std::vector<HybridTensor>& hybrid_tensors(const ruai_model* m) { return m->hy->tensors; }

const HybridTensor* hybrid_tensor(const ruai_model* m, uint64_t id) {
  const auto& t = m->hy->tensors;
  return id >= kTensorBase && id - kTensorBase < t.size() ? &t[id - kTensorBase] : nullptr;
}

const HybridTensor* hybrid_tensor_by_name(const ruai_model* m, const char* name) {
  const auto it = m->hy->by_name.find(name);
  return it == m->hy->by_name.end() ? nullptr : &m->hy->tensors[it->second];
}

namespace {
void add_tensor(Hybrid* y, const std::string& name, size_t rows, size_t cols, float std_dev, float fill) {
  HybridTensor t;
  t.name = name; t.id = kTensorBase + y->tensors.size(); t.rows = rows; t.cols = cols; t.synth_std = std_dev; t.synth_fill = fill;
  y->by_name[name] = y->tensors.size();
  y->tensors.push_back(t);
}
}  // namespace

int hybrid_create(ruai_model* m, const ruai_hybrid_config& cfg, const ruai_layer_config* layers) {
  ruai_ctx* c = m->ctx;
  if (cfg.block > RUAI_BLOCK_SANDWICH) return ruai_fail(c, RUAI_ERR_ARG, "unknown kind of block %u", cfg.block);
  const bool sandwich = cfg.block == RUAI_BLOCK_SANDWICH;
  if (!cfg.vocab_size || !cfg.width || !cfg.num_layers || (!cfg.max_positions && !sandwich)) return ruai_fail(c, RUAI_ERR_SHAPE, "an empty model");
  Hybrid* y = m->hy = new Hybrid();
  y->cfg = cfg;
  y->layers.resize(cfg.num_layers);
  auto tensor = [y](const std::string& name, size_t rows, size_t cols, float std_dev, float fill = 0.0f) { add_tensor(y, name, rows, cols, std_dev, fill); };
  if (sandwich) {
    for (uint32_t l = 0; l < cfg.num_layers; ++l) y->layers[l].cfg = layers[l];
    return sandwich_create(m, add_tensor);
  }
  m->L = cfg.num_layers;
  y->runs.resize(cfg.num_layers);
  for (uint32_t l = 0; l < cfg.num_layers; ++l) y->runs[l].layer = l;
  const uint32_t d = cfg.width;
  tensor("embed", cfg.vocab_size, d, 0.02f);
  tensor("pos", cfg.max_positions, d, 0.02f);
  for (uint32_t l = 0; l < cfg.num_layers; ++l) {
    MixLayer& L = y->layers[l];
    ruai_layer_config f = layers[l];
    const std::string p = "l" + std::to_string(l) + ".", x = p + "mix.";
    if (f.mixer == RUAI_MIX_WKV) f.vdim = f.dim;
    if (f.experts || f.ff_act != RUAI_FF_GELU || f.mixer > RUAI_MIX_HGRN2)
      return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "layer %u: this mixer or feed-forward belongs to blocks of the other kind", l);
    if (!f.heads || !f.dim || !f.vdim) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: heads %u, dim %u, vdim %u", l, f.heads, f.dim, f.vdim);
    L.cfg = f;
    const size_t hk = (size_t)f.heads * f.dim, hv = (size_t)f.heads * f.vdim;
    tensor(p + "norm1", 1, 1, 0.0f, 1.0f);
    tensor(p + "shift", 1, d, 0.0f, 0.5f);
    switch (f.mixer) {
      case RUAI_MIX_DIFF_ATTENTION:
        if (!f.kv_heads || f.heads % f.kv_heads) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: heads %u must be a multiple of kv_heads %u", l, f.heads, f.kv_heads);
        if (!f.window) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: a window of 0 positions sees nothing", l);
        tensor(x + "q", 2 * hk, d, 0.02f);
        tensor(x + "k", 2 * (size_t)f.kv_heads * f.dim, d, 0.02f);
        tensor(x + "v", (size_t)f.kv_heads * f.vdim, d, 0.02f);
        tensor(x + "q.norm", 1, f.dim, 0.0f, 1.0f);
        tensor(x + "k.norm", 1, f.dim, 0.0f, 1.0f);
        for (const char* n : {"lq1", "lk1", "lq2", "lk2"}) tensor(x + n, 1, f.dim, 0.1f);
        break;
      case RUAI_MIX_WKV:
        if (!f.rank) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: the decay projection has rank 0", l);
        for (const char* n : kMuNames) tensor(x + "mu." + n, 1, d, 0.0f, 0.5f);
        for (const char* n : {"r", "k", "v", "g"}) tensor(x + n, hk, d, 0.02f);
        tensor(x + "w1", f.rank, d, 0.02f);
        tensor(x + "w2", hk, f.rank, 0.02f);
        tensor(x + "w0", 1, hk, 0.0f, -2.0f);
        tensor(x + "u", f.heads, f.dim, 0.3f);
        tensor(x + "norm", 1, hk, 0.0f, 1.0f);
        break;
      case RUAI_MIX_HGRN2:
        tensor(x + "q", hk, d, 0.02f);
        tensor(x + "f", hk, d, 0.02f);
        tensor(x + "f.b", 1, hk, 0.0f, 1.0f);
        tensor(x + "lower", 1, hk, 0.0f, 0.5f);
        tensor(x + "v", hv, d, 0.02f);
        tensor(x + "norm", 1, f.vdim, 0.0f, 1.0f);
        break;
      default: return ruai_fail(c, RUAI_ERR_ARG, "layer %u: unknown mixer %u", l, f.mixer);
    }
    tensor(x + "o", d, hv, 0.02f);
    if (f.ff) {
      tensor(p + "mlp.gate", f.ff, d, 0.02f);
      tensor(p + "mlp.up", f.ff, d, 0.02f);
      tensor(p + "mlp.down", d, f.ff, 0.02f);
    }
  }
  tensor("final.norm", 1, 1, 0.0f, 1.0f);
  tensor("head", cfg.vocab_size, d, 0.02f);
  return RUAI_OK;
}

void hybrid_destroy(ruai_model* m) {
  Hybrid* y = m->hy;
  if (!y) return;
  for (MixLayer& L : y->layers) {
    for (DevBuf* b : {&L.norm, &L.shift, &L.q_norm, &L.k_norm, &L.lambda, &L.lower, &L.f_bias, &L.w0, &L.u, &L.head_norm, &L.correction, &L.sink, &L.a_log,
                      &L.conv[0], &L.conv[1], &L.conv[2], &L.n1.w, &L.n1.b, &L.n1b.w, &L.n1b.b, &L.n2.w, &L.n2.b, &L.n2b.w, &L.n2b.b})
      b->release();
    for (DevBuf& b : L.mu) b.release();
    for (Lin& l : L.proj) free_lin(l);
    for (Lin* l : {&L.w2, &L.up, &L.od, &L.o, &L.down, &L.router, &L.uk, &L.uk_t, &L.uv}) free_lin(*l);
  }
  for (MixRun& r : y->runs) { r.state.release(); r.history.release(); }
  for (RotTable& t : y->tables) { t.freq.release(); t.table.release(); }
  free_lin(y->loop_in);
  for (DevBuf* b : {&y->final_norm, &y->final_bias, &y->shift_state, &y->shift_next, &y->h, &y->proj, &y->low, &y->qn, &y->rec_o, &y->cat, &y->hx,
                    &y->span_scratch, &y->span_counters, &y->arg_slots, &y->pass_in, &y->y, &y->hid, &y->q_abs, &y->lat, &y->scores, &y->chosen, &y->weight,
                    &y->place, &y->source, &y->tile_expert, &y->xs, &y->lat_rows, &y->k_all, &y->v_all})
    b->release();
  for (DevBuf& b : y->mix) b.release();
  delete y;
  m->hy = nullptr;
}

int hybrid_build(ruai_model* m, uint32_t bits) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  if (bits != 16 && bits != 32) return model_fail(m, RUAI_ERR_UNSUPPORTED, "a model built from a list of layers runs unquantized: bits 16 (bf16) or 32 (f32), got %u", bits);
  y->act = bits == 16 ? RUAI_BF16 : RUAI_F32;
  if (y->sandwich()) return sandwich_build(m, bits);
  const uint32_t d = m->d;
  uint32_t cat = 0, low = 0;
  for (uint32_t l = 0; l < m->L; ++l) {
    MixLayer& L = y->layers[l];
    const ruai_layer_config& f = L.cfg;
    const std::string p = "l" + std::to_string(l) + ".", x = p + "mix.";
    const uint32_t hk = f.heads * f.dim, hv = f.heads * f.vdim;
    RUAI_TRY(hybrid_move_vec(m, p + "norm1", &L.norm));
    RUAI_TRY(hybrid_move_vec(m, p + "shift", &L.shift));
    if (L.diff()) {
      const uint32_t nq = 2 * hk, nk = 2 * f.kv_heads * f.dim, nv = f.kv_heads * f.vdim;
      RUAI_TRY(hybrid_build_dense(m, &L.proj[0], nq + nk + nv, d, bits, {{x + "q", 0, 1, 0}, {x + "k", nq, 1, 0}, {x + "v", nq + nk, 1, 0}}));
      RUAI_TRY(hybrid_move_vec(m, x + "q.norm", &L.q_norm));
      RUAI_TRY(hybrid_move_vec(m, x + "k.norm", &L.k_norm));
      const float* v[4];
      const char* const names[4] = {"lq1", "lk1", "lq2", "lk2"};
      for (int i = 0; i < 4; ++i) RUAI_TRY(hybrid_take(m, x + names[i], &v[i]));
      RUAI_TRY(L.lambda.alloc(c, sizeof(float)));
      RUAI_TRY(ruai_diff_lambda(c, v[0], v[1], v[2], v[3], f.dim, f.diff, L.lambda.as<float>()));
      RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
      for (const char* n : names) staged_drop(m, id_of(m, x + n));
    } else if (f.mixer == RUAI_MIX_WKV) {
      for (int i = 0; i < MU_N; ++i) RUAI_TRY(hybrid_move_vec(m, x + "mu." + kMuNames[i], &L.mu[i]));
      for (int i = 0; i < 4; ++i) RUAI_TRY(hybrid_build_dense(m, &L.proj[i], hk, d, bits, {{x + kMuNames[i], 0, 1, 0}}));
      RUAI_TRY(hybrid_build_dense(m, &L.proj[MU_W], f.rank, d, bits, {{x + "w1", 0, 1, 0}}));
      RUAI_TRY(hybrid_build_dense(m, &L.w2, hk, f.rank, bits, {{x + "w2", 0, 1, 0}}));
      RUAI_TRY(hybrid_move_vec(m, x + "w0", &L.w0));
      RUAI_TRY(hybrid_move_vec(m, x + "u", &L.u));
      RUAI_TRY(hybrid_move_vec(m, x + "norm", &L.head_norm));
      low = std::max(low, f.rank);
    } else {
      RUAI_TRY(hybrid_build_dense(m, &L.proj[0], hk, d, bits, {{x + "q", 0, 1, 0}}));
      RUAI_TRY(hybrid_build_dense(m, &L.proj[1], hk, d, bits, {{x + "f", 0, 1, 0}}));
      RUAI_TRY(hybrid_build_dense(m, &L.proj[2], hv, d, bits, {{x + "v", 0, 1, 0}}));
      RUAI_TRY(hybrid_move_vec(m, x + "f.b", &L.f_bias));
      RUAI_TRY(hybrid_move_vec(m, x + "lower", &L.lower));
      RUAI_TRY(hybrid_move_vec(m, x + "norm", &L.head_norm));
    }
    if (f.ff) {
      RUAI_TRY(hybrid_build_dense(m, &L.up, 2 * f.ff, d, bits, {{p + "mlp.gate", 0, 2, 0}, {p + "mlp.up", 1, 2, 0}}));
      RUAI_TRY(hybrid_build_dense(m, &L.od, d, hv + f.ff, bits, {{x + "o", 0, 1, 0}, {p + "mlp.down", 0, 1, hv}}));
    } else {
      RUAI_TRY(hybrid_build_dense(m, &L.od, d, hv, bits, {{x + "o", 0, 1, 0}}));
    }
    cat = std::max(cat, hv + f.ff);
  }
  RUAI_TRY(hybrid_move_vec(m, "embed", &m->embed));
  RUAI_TRY(hybrid_move_vec(m, "pos", &m->wpe));
  RUAI_TRY(hybrid_move_vec(m, "final.norm", &y->final_norm));
  RUAI_TRY(hybrid_build_dense(m, &m->head, m->V, d, bits, {{"head", 0, 1, 0}}));
  y->ldd = hy_up8(d); y->ldcat = hy_up8(cat); y->ldlow = hy_up8(low);
  return RUAI_OK;
}

void hybrid_cache_shape(const ruai_model* m, uint32_t run, uint32_t* heads, uint32_t* kw, uint32_t* vw) {
  const MixLayer& L = m->hy->layers[m->hy->runs[run].layer];
  if (L.latent()) {  // one row per position for all heads: the latent and the rotated key part
    *heads = 1; *kw = L.kdp() + L.rotp(); *vw = 0;
    return;
  }
  *heads = L.attention() ? L.cfg.kv_heads : 0;
  *kw = 2 * L.kdp();
  *vw = L.vdp();
}

int hybrid_positions(ruai_model* m, uint32_t positions) {
  for (RotTable& t : m->hy->tables) {
    if (t.rows >= positions) continue;
    t.rows = 0;
    RUAI_TRY(t.table.alloc(m->ctx, (size_t)positions * (t.cfg.rot / 2) * sizeof(float2)));
    RUAI_TRY(ruai_rotary_table(m->ctx, t.freq.as<double>(), t.cfg.dims / 2, t.cfg.rot / 2, positions, t.scale, t.table.as<float2>()));
    t.rows = positions;
    drop_graph(m);
  }
  return RUAI_OK;
}

int hybrid_state_alloc(ruai_model* m, uint32_t B) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
  auto zeroed = [&](DevBuf& b, size_t n) -> int {
    RUAI_TRY(b.alloc(c, n));
    RUAI_CUDA(c, cudaMemsetAsync(b.p, 0, n, c->stream));
    return RUAI_OK;
  };
  if (!y->sandwich()) {
    const size_t shift = (size_t)m->L * B * 2 * m->d * sizeof(float);
    RUAI_TRY(zeroed(y->shift_state, shift));
    RUAI_TRY(zeroed(y->shift_next, shift));
  }
  for (MixRun& r : y->runs) {
    const MixLayer& L = y->layers[r.layer];
    const ruai_layer_config& f = L.cfg;
    if (!L.attention()) RUAI_TRY(zeroed(r.state, (size_t)B * f.heads * f.dim * f.vdim * sizeof(float)));
    if (L.delta()) RUAI_TRY(zeroed(r.history, (size_t)B * f.conv * (2 * f.kv_heads * f.dim + f.heads * f.vdim) * sizeof(float)));
  }
  return RUAI_OK;
}

int hybrid_span_scratch(ruai_model* m, size_t scratch, size_t counters) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  if (scratch <= y->span_scratch.bytes && counters * sizeof(unsigned) <= y->span_counters.bytes) return RUAI_OK;
  RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
  drop_graph(m);
  RUAI_TRY(y->span_scratch.reserve(c, scratch));
  if (counters * sizeof(unsigned) > y->span_counters.bytes) {
    RUAI_TRY(y->span_counters.alloc(c, counters * sizeof(unsigned)));
    RUAI_CUDA(c, cudaMemsetAsync(y->span_counters.p, 0, counters * sizeof(unsigned), c->stream));
  }
  return RUAI_OK;
}

int hybrid_reserve(ruai_model* m, uint32_t rows, uint32_t out_rows, uint32_t B, uint32_t T) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const size_t es = hy_act_bytes(y);
  if (rows > y->rows) {
    RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
    drop_graph(m);
    y->rows = 0;
    size_t proj = 0, qn = 0, rec = 0;
    int mixes = 1;
    for (const MixLayer& L : y->layers) {
      proj = std::max(proj, L.proj_floats());
      if (L.diff()) qn = std::max(qn, (size_t)2 * L.cfg.heads * L.kdp());
      else if (L.latent()) qn = std::max(qn, (size_t)L.cfg.heads * (std::max(L.kdp(), L.dimp()) + L.rotp()));
      else if (!L.delta()) rec = std::max(rec, (size_t)L.cfg.heads * L.cfg.vdim);
      if (L.cfg.mixer == RUAI_MIX_WKV) mixes = MU_N;
    }
    const size_t r = rows;
    RUAI_TRY(m->d_ids.alloc(c, r * sizeof(int32_t)));
    RUAI_TRY(m->x.alloc(c, r * m->d * sizeof(float)));
    RUAI_TRY(y->h.alloc(c, r * y->ldd * es));
    if (!y->sandwich())
      for (int i = 0; i < mixes; ++i) RUAI_TRY(y->mix[i].alloc(c, r * y->ldd * es));
    RUAI_TRY(y->proj.alloc(c, r * proj * sizeof(float)));
    RUAI_TRY(y->low.alloc(c, r * y->ldlow * es));
    RUAI_TRY(y->qn.alloc(c, r * qn * sizeof(float)));
    RUAI_TRY(y->rec_o.alloc(c, r * rec * sizeof(float)));
    RUAI_TRY(y->cat.alloc(c, r * y->ldcat * es));
    if (!y->arg_slots.p) {
      RUAI_TRY(y->arg_slots.alloc(c, 16 * (size_t)kDenseArgSlots * sizeof(unsigned long long)));
      RUAI_CUDA(c, cudaMemsetAsync(y->arg_slots.p, 0, y->arg_slots.bytes, c->stream));
    }
    y->rows = rows;
  }
  if (out_rows > y->out_rows) {
    RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
    drop_graph(m);
    y->out_rows = 0;
    RUAI_TRY(m->logits.alloc(c, (size_t)out_rows * m->V * sizeof(float)));
    RUAI_TRY(m->xl.alloc(c, (size_t)out_rows * m->d * sizeof(float)));
    RUAI_TRY(y->hx.alloc(c, (size_t)out_rows * y->ldd * es));
    y->out_rows = out_rows;
  }
  if (y->sandwich()) return sandwich_reserve(m, rows, B, T);
  size_t scratch = 0, counters = 0;
  for (uint32_t l = 0; l < m->L; ++l) {
    if (!y->layers[l].attention()) continue;
    size_t n;
    scratch = std::max(scratch, ruai_attn_span_scratch(span_params(m, l, B, T), B, &n));
    counters = std::max(counters, n);
  }
  return hybrid_span_scratch(m, scratch, counters);
}

int hybrid_issue(ruai_model* m, uint32_t B, uint32_t T, const HeadRows& head, bool want_argmax) {
  Hybrid* y = m->hy;
  if (y->sandwich()) return sandwich_issue(m, B, T, head, want_argmax);
  ruai_ctx* c = m->ctx;
  const uint32_t rows = B * T, d = m->d;
  int32_t* len = m->d_len.as<int32_t>();
  float* x = m->x.as<float>();
  RUAI_TRY(ruai_embed(c, m->d_ids.as<int32_t>(), m->embed.as<float>(), m->wpe.as<float>(), len, rows, T, d, m->V, x, m->d_err.as<int>(), nullptr));
  for (uint32_t l = 0; l < m->L; ++l) {
    MixLayer& L = y->layers[l];
    const ruai_layer_config& f = L.cfg;
    TokenMixParams tm;
    tm.x = x; tm.g = L.norm.as<float>(); tm.eps = m->eps; tm.T = T; tm.d = d; tm.len = len; tm.shift = L.shift.as<float>();
    const size_t at = (size_t)l * B * 2 * d;
    tm.state = y->shift_state.as<float>() + at;
    tm.state_out = (T == 1 ? y->shift_state : y->shift_next).as<float>() + at;
    tm.h_out = f.ff ? y->h.p : nullptr;
    tm.ld = y->ldd; tm.out_dtype = y->act;
    tm.mix_out[0] = y->mix[0].p;
    if (f.mixer == RUAI_MIX_WKV) {
      tm.n_mix = MU_N;
      for (int i = 0; i < MU_N; ++i) { tm.mix_out[i] = y->mix[i].p; tm.mu[i] = L.mu[i].as<float>(); }
    }
    RUAI_TRY(ruai_token_mix(c, tm, B));
    RUAI_TRY(issue_projections(m, l, rows, T));
    float* proj = y->proj.as<float>();
    if (L.diff()) {
      SpanParams p = span_params(m, l, B, T);
      p.qkv = proj; p.q = y->qn.as<float>();
      p.out = y->cat.p; p.out_ld = y->ldcat; p.out_dtype = y->act;
      p.scratch = y->span_scratch.as<float>(); p.counters = y->span_counters.as<unsigned>();
      RUAI_TRY(ruai_attn_span(c, p, B));
    } else {
      const uint32_t hk = hy_up4(f.heads * f.dim);
      const size_t sec = (size_t)rows * hk;
      RecurrenceParams p;
      p.r = proj; p.ld_r = hk; p.ld_k = hk; p.ld_w = hk;
      if (f.mixer == RUAI_MIX_WKV) {
        p.k = proj + sec; p.v = proj + 2 * sec; p.ld_v = hk; p.gate = proj + 3 * sec; p.ld_gate = hk;
        if (T > 1) p.w = proj + 4 * sec;
        p.w2 = L.w2.w->data; p.w2_bits = (int)L.w2.w->bits; p.w2_ld = L.w2.w->ld; p.rank = f.rank; p.w0 = L.w0.as<float>();
        p.t = y->low.p; p.t_dtype = y->act; p.ld_t = y->ldlow;
        p.u = L.u.as<float>();
        p.norm_per_head = 1;
      } else {
        p.w = proj + sec; p.v = proj + 2 * sec; p.ld_v = hy_up4(f.heads * f.vdim);
      }
      p.state = y->runs[l].state.as<float>(); p.len = len; p.T = T; p.H = f.heads; p.dk = f.dim; p.dv = f.vdim;
      p.o = y->rec_o.as<float>();
      p.eps = m->eps; p.norm = L.head_norm.as<float>();
      p.out = y->cat.p; p.out_ld = y->ldcat; p.out_dtype = y->act;
      RUAI_TRY(ruai_recurrence(c, p, B));
    }
    RUAI_TRY(issue_output(m, l, rows, x));
  }
  if (T > 1)
    RUAI_CUDA(c, cudaMemcpyAsync(y->shift_state.p, y->shift_next.p, (size_t)m->L * B * 2 * d * sizeof(float), cudaMemcpyDeviceToDevice, c->stream));
  const uint32_t out_rows = head.count(B, T);
  if (out_rows == 0) return ruai_add_scalar(c, len, (int32_t)T);
  const float* hx = x;
  TokenMixParams fn;
  if (head.mode == HeadRows::LIST) fn.rows = m->d_rows.as<int32_t>();
  else if (head.mode == HeadRows::LAST && T > 1) {
    RUAI_TRY(ruai_take_last_rows(c, x, B, T, d, m->xl.as<float>()));
    hx = m->xl.as<float>();
  }
  fn.x = hx; fn.g = y->final_norm.as<float>(); fn.eps = m->eps; fn.T = out_rows; fn.d = d; fn.mix_out[0] = y->hx.p; fn.ld = y->ldd; fn.out_dtype = y->act;
  RUAI_TRY(ruai_token_mix(c, fn, 1));
  const bool pick = want_argmax && out_rows <= 16;
  RUAI_TRY(hybrid_issue_head(m, out_rows, pick, T));
  if (!pick) {
    RUAI_TRY(ruai_add_scalar(c, len, (int32_t)T));
    if (want_argmax) RUAI_TRY(ruai_argmax(c, m->logits.as<float>(), m->V, out_rows, m->V, m->d_ids.as<int32_t>(), 0));
  }
  return RUAI_OK;
}

// The matrix products of one step of B tokens and nothing else (their inputs are whatever the buffers hold).
int hybrid_time_linears(ruai_model* m, uint32_t B, uint32_t iters, float* ms_total, uint32_t* launches, double* bytes_per_pass) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const size_t es = hy_act_bytes(y);
  for (DevBuf* b : {&y->h, &y->mix[0], &y->mix[1], &y->mix[2], &y->mix[3], &y->mix[4], &y->cat, &y->hx, &m->x, &y->low, &y->proj, &y->lat, &y->hid, &y->pass_in})
    if (b->p) RUAI_CUDA(c, cudaMemsetAsync(b->p, 0, b->bytes, c->stream));
  double bytes = 0.0;
  const unsigned long long before = c->launches;
  unsigned long long per_pass = 0;
  auto pass = [&]() -> int {
    if (y->sandwich()) {
      RUAI_TRY(sandwich_issue_linears(m, B));
      return hybrid_issue_head(m, B, false, 0);
    }
    for (uint32_t l = 0; l < m->L; ++l) {
      RUAI_TRY(issue_projections(m, l, B, 1));
      RUAI_TRY(issue_output(m, l, B, m->x.as<float>()));
    }
    return hybrid_issue_head(m, B, false, 0);
  };
  RUAI_TRY(pass());
  per_pass = c->launches - before;
  if (y->sandwich()) bytes = sandwich_linear_bytes(m, B);
  else for (MixLayer& L : y->layers)
    for (const Lin* w : {&L.proj[0], &L.proj[1], &L.proj[2], &L.proj[3], &L.proj[4], &L.up, &L.od})
      if (w->w) bytes += w->bytes() + (double)B * (es * w->w->k + 4.0 * w->w->n);
  bytes += m->head.bytes() + (double)B * (es * m->head.w->k + 4.0 * m->head.w->n);
  RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
  RUAI_CUDA(c, cudaEventRecord(c->ev0, c->stream));
  for (uint32_t i = 0; i < iters; ++i) RUAI_TRY(pass());
  RUAI_CUDA(c, cudaEventRecord(c->ev1, c->stream));
  RUAI_CUDA(c, cudaEventSynchronize(c->ev1));
  RUAI_CUDA(c, cudaEventElapsedTime(ms_total, c->ev0, c->ev1));
  if (launches) *launches = (uint32_t)per_pass;
  if (bytes_per_pass) *bytes_per_pass = bytes;
  return RUAI_OK;
}

double hybrid_step_bytes(const ruai_model* m, uint32_t B, uint32_t len) {
  const Hybrid* y = m->hy;
  if (y->sandwich()) return sandwich_step_bytes(m, B, len);
  double w = m->head.bytes() + 4.0, per_seq = 4.0 * m->d * 2;
  for (const MixLayer& L : y->layers) {
    for (const Lin* l : {&L.proj[0], &L.proj[1], &L.proj[2], &L.proj[3], &L.proj[4], &L.w2, &L.up, &L.od}) w += l->bytes();
    for (const DevBuf* b : {&L.norm, &L.shift, &L.q_norm, &L.k_norm, &L.lower, &L.f_bias, &L.w0, &L.u, &L.head_norm, &L.mu[0], &L.mu[1], &L.mu[2], &L.mu[3], &L.mu[4]})
      w += (double)b->bytes;
    per_seq += 2.0 * 2 * m->d * 4.0;  // the previous token's values, read and written
    if (L.attention()) {
      const uint64_t span = std::min<uint64_t>(len + 1, (uint64_t)L.cfg.window + L.cfg.keep_first);
      per_seq += (double)(span + 1) * L.cfg.kv_heads * (2 * L.cfg.dim + L.cfg.vdim) * 4.0;
    } else {
      per_seq += 2.0 * L.cfg.heads * L.cfg.dim * L.cfg.vdim * 4.0;
    }
  }
  return w + B * per_seq;
}
