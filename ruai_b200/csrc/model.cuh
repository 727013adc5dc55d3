// Device state of a model: weights, KV cache, activations, the captured decode step.
#pragma once
#include <map>
#include <vector>

#include "common.cuh"
#include "pstep.cuh"
#include "tp.cuh"

struct DevBuf {
  void* p = nullptr;
  size_t bytes = 0;
  int alloc(ruai_ctx* c, size_t n) {
    release();
    RUAI_CUDA(c, cudaMalloc(&p, n ? n : 1));
    bytes = n;
    return RUAI_OK;
  }
  int reserve(ruai_ctx* c, size_t n) { return n <= bytes && p ? RUAI_OK : alloc(c, n); }
  void release() {
    if (p) cudaFree(p);
    p = nullptr;
    bytes = 0;
  }
  template <typename T> T* as() const { return (T*)p; }
};

// A reference Linear after quantize_int8 / quantize_int4: full (unsharded) buffers in the
// reference layout, on the device.  Lives only while a layer is being loaded.
struct RefQ {
  uint32_t k = 0, n = 0, bits = 0, group = 0;
  DevBuf q, scale;
  uint32_t q_rows() const { return bits == 8 ? k : k / 2; }
  uint32_t s_rows() const { return bits == 8 ? 1 : k / group; }
  RefQ() = default;
  RefQ(const RefQ&) = delete;
  RefQ& operator=(const RefQ&) = delete;
  ~RefQ() { q.release(); scale.release(); }
};

struct Lin {
  ruai_qweight* w = nullptr;
  ruai_sweight sw;  // the same weight in the tile-stream layout of the persistent decode kernel (Llama only)
  DevBuf bias;
  double bytes() const { return w ? (double)w->k * w->n * w->bits / 8.0 + (double)w->scale_bytes + (double)bias.bytes : 0.0; }
};

struct Layer {
  DevBuf n1w, n1b, n2w, n2b;
  Lin qkv, o, up, down;  // up = gate/up interleaved (Llama) or c_fc (GPT-2)
  DevBuf kc, vc;         // KV cache [B, KVl, cap, hd]
};

// Device state of the persistent decode step (pstep.cu).
struct PStep {
  bool tried = false, usable = false;
  int wanted = -1;  // -1: the environment decides (RUAI_B200_PSTEP=1 turns it on), 0 / 1: ruai_model_use_persistent_step
  DevBuf layers, x, ss, acc, poison, att_part, arg_slots, sync;  // sync: [0] barrier counter, [1] abort flag
  unsigned bar_base = 0;
  uint32_t table_cap = 0, table_B = 0, splits = 0, att_rows = 0;
  size_t acc_elems = 0;
};

struct Hybrid;  // hybrid.cuh

struct ruai_model {
  ruai_ctx* ctx = nullptr;
  bool llama = true;
  Hybrid* hy = nullptr;  // a decoder built from a list of layers; `llama` is false then
  ruai_llama_config lc{};
  ruai_gpt2_config gc{};
  uint32_t L = 0, d = 0, H = 0, KV = 0, hd = 0, ffn = 0, V = 0, max_pos = 0;
  uint32_t rank = 0, world = 1, Hl = 0, KVl = 0, fl = 0, Vl = 0;
  float eps = 1e-5f;
  bool tied = false;
  // weights
  DevBuf embed, wpe, final_w, final_b, rope_table;
  std::vector<Layer> layers;
  Lin head;
  bool quantized = false;
  uint32_t bits = 0, group = 0;
  std::map<uint64_t, DevBuf> staged;  // f32 tensors set before quantizing
  std::map<uint64_t, RefQ*> staged_q; // Linears that arrived already quantized (a checkpoint in the reference's format)
  // cache state
  uint32_t B = 0, len = 0, cap = 0;
  // device state
  DevBuf d_ids, d_rows, d_len, d_err, x, xn, qkv, att, hbuf, xl, logits, attn_scratch, attn_counters, sumsq, arg_slots, arg_counter;
  uint32_t act_rows = 0, logit_rows = 0;
  // decode graph
  cudaGraphExec_t graph = nullptr;
  uint32_t graph_B = 0, graph_cap = 0, graph_launches = 0;
  unsigned long long graph_epoch = 0;  // the context's scratch_epoch at capture: the graph holds the scratch's address
  bool len_dirty = true;  // the device copy of `len` may differ from the host's
  PStep ps;
  ruai_tp_state tp;
};

int model_fail(ruai_model* m, int code, const char* fmt, ...);
void drop_graph(ruai_model* m);
// An f32 tensor set before the weights are built: lookup, removal, allocation.
int staged_get(ruai_model* m, uint64_t id, DevBuf** out);
void staged_drop(ruai_model* m, uint64_t id);
int stage_alloc(ruai_model* m, uint64_t id, size_t count, DevBuf** out);

// Which rows of a step get logits: all B*T, the last of each sequence, or a list.
struct HeadRows {
  enum Mode { LAST, ALL, LIST } mode = LAST;
  uint32_t n = 0;  // LIST: how many (the list is in ruai_model::d_rows)
  uint32_t count(uint32_t B, uint32_t T) const { return mode == ALL ? B * T : mode == LAST ? B : n; }
};
