// State of a loaded model behind the C ABI: configuration, weights, KV caches, the token loop's device
// words and the captured decode step. Shared by the Llama-2 driver (model.cu) and the layer-list decoder
// designs (decoder.cu), which plug their pass over T tokens into the same loop.
#pragma once
#include <memory>
#include <string>
#include <vector>

#include "decoder.h"
#include "runtime.h"

namespace vkl {
struct Layer {
  vkl_tensor *attn_norm = nullptr, *ffn_norm = nullptr;
  vkl_tensor *wq = nullptr, *wk = nullptr, *wv = nullptr, *wo = nullptr;
  vkl_tensor *gate = nullptr, *up = nullptr, *down = nullptr;
  vkl_tensor *kcache = nullptr, *vcache = nullptr;
  // recurrent layers: state per head [heads][value][key] in fp32, the last projections before the convolution
  vkl_tensor *state = nullptr, *ring = nullptr;
};

// Optional per-kernel timing of a pass: an event after every launch, tagged with
// the kernel's class (0 embedding, 1 norm+QKV, 2 attention, 3 o_proj, 4 gate/up,
// 5 down, 6 lm head, 7 arg-max, 8 recurrent layers' steps between the projections, 9 norms of their own).
struct Marker {
  std::vector<cudaEvent_t> ev;
  std::vector<int> cls;
  cudaStream_t s;
  void mark(int c) {
    cudaEvent_t e;
    cudaEventCreate(&e);
    cudaEventRecord(e, s);
    ev.push_back(e);
    cls.push_back(c);
  }
};
}  // namespace vkl

struct vkl_model {
  vkl_device *dev = nullptr;
  vkl_model_config cfg;
  cudaStream_t stream = nullptr;
  uint32_t head_dim = 0, heads_l = 0, dim_l = 0, ffn_l = 0, vocab_l = 0;
  std::vector<vkl::Layer> L;  // Llama-2: blocks; a decoder design: layer runs, of which only caches and states live here
  std::unique_ptr<vkl::Decoder> dec;  // set for the layer-list decoder designs
  vkl_tensor *tok_embd = nullptr, *output_norm = nullptr, *output = nullptr;
  vkl_tensor *fc = nullptr, *fs = nullptr;
  // activations, sized for `cap_T` rows
  uint32_t cap_T = 0;
  vkl_tensor *x = nullptr, *xn = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *ao = nullptr, *t = nullptr;
  vkl_tensor *gu32 = nullptr;  // [2, cap_T, ffn] fp32 gate and up results of the FP16 prefill GEMMs
  bool gemm_used = false;      // a tensor-core GEMM ran since the last check of state[6]
  vkl_tensor *logits16 = nullptr, *logits32 = nullptr;
  vkl_tensor *toks = nullptr;  // [cap_T] device token ids; toks[0] is the decode token
  vkl_tensor *state = nullptr; // uint32[8]: [0] pos, [1] step, [2] next id, [3] all-reduces, [4] arg exchanges, [5] forced tokens, [6] GEMM wait error
  vkl_tensor *forced = nullptr;  // prompt ids for token-by-token prefill
  // tensor parallelism: this rank's exchange buffer (plain cudaMalloc so that it can be
  // exported over CUDA IPC) and every rank's mapping of it
  void *tp_buf = nullptr;
  size_t tp_bytes = 0;
  uint32_t tp_flag_off = 0;
  void *tp_peer[8] = {};
  bool tp_connected = false;
  // many-token passes of a sharded model: two alternating regions of fp32 partial sums [tp_pf_rows, dim]
  // and the ranks' flag words behind the one-token exchange area, and the count of all-reduces so far
  size_t tp_pf_off = 0, tp_pf_flag_off = 0;
  uint32_t tp_pf_rows = 0, tp_pf_seq = 0;
  vkl_tensor *out_ids = nullptr;
  vkl_tensor *argpart = nullptr, *attn_scratch = nullptr, *attn_counters = nullptr;
  uint32_t splits = 8, out_cap = 0;
  cudaGraphExec_t decode_graph = nullptr;
  bool use_pdl = true;
  // persistent single-kernel decode step (decode_mega.cu)
  bool mega_ready = false, mega_tried = false;
  int mega_grid = 0;
  vkl_tensor *mega_ops = nullptr, *mega_sync = nullptr, *mega_arg = nullptr, *mega_attn = nullptr, *mega_stages = nullptr, *mega_counts = nullptr, *mega_ll = nullptr;
  std::vector<vkl_tensor *> mega_packed;  // the ops' weight streams in the persistent kernel's layout
  vkl::MegaParams mp;
  uint32_t mega_launches_per_token = 1;
  uint32_t sm_mhz = 0;  // measured SM clock, for the profiled launches' cycle counts
  uint32_t wait_limit = 0;  // polls a wait of the decode kernel may spin (0: the default of build_mega)
  bool tp_failed = false;   // a wait on another rank ran out: the ranks' sequence counters are out of step until they reconnect
  unsigned char *pin = nullptr;  // pinned host staging of the one-token call: this rank's fp32 logits, then the decode kernel's error word
  cudaEvent_t ev0 = nullptr, ev1 = nullptr, ev2 = nullptr;
  uint32_t *pos_dev() { return (uint32_t *)state->data(); }
  uint32_t *step_dev() { return (uint32_t *)state->data() + 1; }
  uint32_t *next_dev() { return (uint32_t *)state->data() + 2; }
  ~vkl_model() {
    if (decode_graph) cudaGraphExecDestroy(decode_graph);
    dec.reset();
    if (tp_buf) cudaFree(tp_buf);
    if (pin) cudaFreeHost(pin);
    for (auto &l : L)
      for (vkl_tensor *p : {l.attn_norm, l.ffn_norm, l.wq, l.wk, l.wv, l.wo, l.gate, l.up, l.down, l.kcache, l.vcache, l.state, l.ring}) vkl_tensor_release(p);
    for (vkl_tensor *p : mega_packed) vkl_tensor_release(p);
    for (vkl_tensor *p : {tok_embd, output_norm, output, fc, fs, x, xn, q, k, v, ao, t, gu32, logits16, logits32, toks, state, out_ids, forced, argpart, attn_scratch, attn_counters, mega_ops, mega_sync, mega_arg, mega_attn, mega_stages, mega_counts, mega_ll})
      vkl_tensor_release(p);
    if (ev0) cudaEventDestroy(ev0);
    if (ev1) cudaEventDestroy(ev1);
    if (ev2) cudaEventDestroy(ev2);
    if (stream) {
      dev->remove_stream(stream);
      cudaStreamDestroy(stream);
    }
  }
};

namespace vkl {
// What every architecture's model needs: stream, events, logits, loop state, id buffers. cfg is set.
int model_init_common(vkl_model *m);
// New weights or buffers: a captured decode step is stale.
void model_drop_graph(vkl_model *m);
}  // namespace vkl
