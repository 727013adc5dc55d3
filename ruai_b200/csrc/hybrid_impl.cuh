// Inside of the decoder built from a list of layers: shared by hybrid.cu and hybrid_sandwich.cu.
#pragma once
#include "attn_latent.cuh"
#include "attn_span.cuh"
#include "delta.cuh"
#include "hybrid.cuh"
#include "moe.cuh"
#include "recurrence.cuh"
#include "resid_norm.cuh"
#include "token_mix.cuh"

inline uint32_t hy_up4(uint32_t v) { return (v + 3) & ~3u; }
inline uint32_t hy_up8(uint32_t v) { return (v + 7) & ~7u; }

enum { MU_R, MU_K, MU_V, MU_G, MU_W, MU_N };

struct NormBufs { DevBuf w, b; };

struct MixLayer {
  ruai_layer_config cfg{};
  // weights
  DevBuf norm, shift, q_norm, k_norm, lambda, lower, f_bias, mu[MU_N], w0, u, head_norm;
  // attention: [0] = q | k | v;  wkv: r, k, v, g, w1;  hgrn2: q, f, v;  latent: q, dkv, g;  delta: q, k, v, b, a, g
  Lin proj[6];
  Lin w2, up, od;  // up: gate / up rows interleaved (of one expert after the other); od: W_o and W_down side by side along k
  // sandwich blocks: mixer and feed-forward have outputs of their own
  NormBufs n1, n1b, n2, n2b;
  Lin o, down, router;
  DevBuf correction;
  uint32_t router_parts = 1;  // the router's matrix product is cut into so many along its inputs
  Lin uk, uk_t, uv;  // latent: keys [heads * dimp, rank], the same per head transposed [heads * rank, dim], values [heads * vdp, rank]
  DevBuf sink;
  uint32_t table = 0;  // which rotation table
  DevBuf conv[3], a_log;

  uint32_t kdp() const { return hy_up4(latent() ? cfg.rank : cfg.dim); }
  uint32_t vdp() const { return hy_up4(cfg.vdim); }
  uint32_t mix_width() const { return cfg.heads * cfg.vdim; }  // what W_o reads
  bool diff() const { return cfg.mixer == RUAI_MIX_DIFF_ATTENTION; }
  bool latent() const { return cfg.mixer == RUAI_MIX_LATENT; }
  bool delta() const { return cfg.mixer == RUAI_MIX_DELTA; }
  bool attention() const { return diff() || latent(); }  // caches keys
  // latent: a head's query, and a row of the projections
  uint32_t dimp() const { return hy_up4(cfg.dim); }
  uint32_t rotp() const { return hy_up4(cfg.rot_dim); }
  uint32_t qh() const { return dimp() + rotp(); }
  uint32_t lat_ld() const { return hy_up4(cfg.heads * qh() + cfg.rank + cfg.rot_dim); }
  // f32 floats per token of the projections' results
  size_t proj_floats() const {
    const uint32_t hk = hy_up4(cfg.heads * cfg.dim), hv = hy_up4(cfg.heads * cfg.vdim);
    if (diff()) return qkv_ld();
    if (latent()) return lat_ld() + hy_up4(cfg.heads);
    if (delta()) return 2 * (size_t)hy_up4(cfg.kv_heads * cfg.dim) + 2 * (size_t)hv + 2 * (size_t)hy_up4(cfg.heads);
    if (cfg.mixer == RUAI_MIX_WKV) return 5 * (size_t)hk;  // r, k, v, gate, decay
    return 2 * (size_t)hk + hv;
  }
  uint32_t qkv_ld() const { return hy_up4(2 * cfg.dim * (cfg.heads + cfg.kv_heads) + cfg.kv_heads * cfg.vdim); }
};

// One pass through a layer: its weights may serve several, its cache (ruai_model::layers) and states are its own.
struct MixRun {
  uint32_t layer = 0;
  bool pass_begins = false;  // the stream meets the embedding again first
  DevBuf state;              // recurrent state
  DevBuf history;            // last inputs of the convolutions
};

struct RotTable {
  RotaryConfig cfg;
  double scale = 1.0;
  DevBuf freq, table;
  uint32_t rows = 0;
};

struct Hybrid {
  ruai_hybrid_config cfg{};
  std::vector<MixLayer> layers;
  std::vector<MixRun> runs;
  std::vector<HybridTensor> tensors;
  std::map<std::string, size_t> by_name;
  std::vector<RotTable> tables;
  DevBuf final_norm, final_bias;
  Lin loop_in;
  int act = RUAI_BF16;  // type of the matrix products' inputs
  // per sequence: h and its shifted form of the last token, [L][B][2][d]; a step of several tokens writes the second
  DevBuf shift_state, shift_next;
  // activations
  DevBuf h, mix[MU_N], proj, low, qn, rec_o, cat, hx, span_scratch, span_counters, arg_slots;
  uint32_t rows = 0, out_rows = 0;
  uint32_t ldd = 0, ldcat = 0, ldlow = 0;
  // sandwich blocks
  DevBuf pass_in, y, hid, q_abs, lat, scores, chosen, weight, place, source, tile_expert, xs;
  DevBuf lat_rows, k_all, v_all;  // keys and values of every position, where a step of many tokens spreads them out
  uint32_t ldff = 0, ldpass = 0;
  bool sandwich() const { return cfg.block == RUAI_BLOCK_SANDWICH; }
};

inline size_t hy_act_bytes(const Hybrid* y) { return y->act == RUAI_F32 ? 4 : 2; }

// ---- hybrid.cu ----
int hybrid_take(ruai_model* m, const std::string& name, const float** out);
int hybrid_move_vec(ruai_model* m, const std::string& name, DevBuf* dst);
// Rows [src0, src0 + rows) (rows 0: all) of a tensor to rows row0, row0 + row_step, ... of a weight, at column col0.
struct RowPart { std::string name; uint32_t row0, row_step, col0, src0 = 0, rows = 0; };
int hybrid_build_dense(ruai_model* m, Lin* out, uint32_t n, uint32_t k, uint32_t bits, const std::vector<RowPart>& parts);
int hybrid_drop(ruai_model* m, const std::string& name);
// Scratch of the few-queries attention.
int hybrid_span_scratch(ruai_model* m, size_t scratch, size_t counters);
int hybrid_issue_head(ruai_model* m, uint32_t out_rows, bool pick, uint32_t len_add);

// ---- hybrid_sandwich.cu ----
typedef void (*HybridTensorFn)(Hybrid* y, const std::string& name, size_t rows, size_t cols, float std_dev, float fill);
int sandwich_create(ruai_model* m, HybridTensorFn tensor);
int sandwich_build(ruai_model* m, uint32_t bits);
int sandwich_reserve(ruai_model* m, uint32_t rows, uint32_t B, uint32_t T);
int sandwich_issue(ruai_model* m, uint32_t B, uint32_t T, const HeadRows& head, bool want_argmax);
// The matrix products of a step of B tokens alone; bytes: of one pass.
int sandwich_issue_linears(ruai_model* m, uint32_t B);
double sandwich_linear_bytes(const ruai_model* m, uint32_t B);
double sandwich_step_bytes(const ruai_model* m, uint32_t B, uint32_t len);
