// decoder.h — the decoder object, shared by decoder.cu (entry points, the attention-only layer walk)
// and decoder_mixed.cu (decoders whose layers carry different sequence mixers).
#pragma once

#include <map>
#include <memory>
#include <string>
#include <vector>

#include "kernels.h"

namespace cg {

struct MixedModel;

struct Layer {
  cg_tensor *w_qkv = nullptr, *w_o = nullptr, *w_gu = nullptr, *w_down = nullptr;
  cg_tensor *ln_in = nullptr, *ln_post_attn = nullptr, *ln_pre_ffn = nullptr, *ln_post_ffn = nullptr;
  cg_tensor *q_norm = nullptr, *k_norm = nullptr;
  cg_tensor *k_cache = nullptr, *v_cache = nullptr;
  // mixture-of-experts layers (qwen3.rs:64-133): router [E, H] f32, this rank's experts stacked
  bool moe = false;
  cg_tensor *router = nullptr, *router3 = nullptr, *we_gate = nullptr, *we_up = nullptr, *we_down = nullptr;
};

inline void drop(cg_tensor*& t) {
  if (t) release(t);
  t = nullptr;
}

}  // namespace cg

struct cg_decoder {
  cg_ctx* c = nullptr;
  cg_decoder_config cfg{};
  std::map<std::string, cg_tensor*> params;  // as handed over, until finalize
  bool finalized = false;
  // sharded sizes
  int nh = 0, nkv = 0, d = 0, F = 0, Vp = 0, H = 0, qkv = 0;
  std::vector<cg::Layer> layers;
  cg_tensor *embed = nullptr, *head = nullptr, *ln_f = nullptr;
  cg_tensor *cos_t = nullptr, *sin_t = nullptr;
  cg_tensor *cos_l = nullptr, *sin_l = nullptr;  // tables of the second rope base (gemma3.rs:154-159), or null
  // state
  cg_tensor* state = nullptr;     // int64[2] on device: {position, tokens generated}
  cg_tensor* cur = nullptr;       // u32 [B]: the tokens the next step consumes
  cg_tensor* history = nullptr;   // u32 [max_batch, max_seq]
  cg_tensor* logits = nullptr;    // f32 [tp_world, B, Vp]
  int64_t B = 0, pos = 0, generated = 0;
  // workspace (sized for `cap` tokens)
  int64_t cap = 0;
  cg_tensor *x = nullptr, *xn = nullptr, *qkvb = nullptr, *q = nullptr, *att = nullptr, *hact = nullptr,
            *tmp = nullptr, *xl = nullptr, *splitk = nullptr, *best = nullptr;
  // mixture-of-experts scratch, sized for cap * top_k pairs
  cg_tensor *m_ids = nullptr, *m_wts = nullptr, *m_pos = nullptr, *m_tiles = nullptr, *m_xg = nullptr, *m_h = nullptr,
            *m_y = nullptr, *m_xs3 = nullptr, *m_logits = nullptr;
  int El = 0;                    // experts on this rank
  int EW = 1, ER = 0;            // ranks the experts are split over, and this rank's place among them
  cg_tensor *ep_x = nullptr, *ep_y = nullptr;  // expert parallelism: every rank's rows gathered / this rank's expert sums for them
  bool pending_reduce = false;   // x still lacks the addends pushed by the last row-parallel GEMM
  // norm hand-over (see DecGemm): xn holds bf16(x * gain) un-normalised and ss the per-CTA sums
  // of squares the last residual GEMM wrote; the next GEMM applies 1 / rms in its epilogue
  bool xn_raw = false;
  bool xn_ready = false;         // xn already holds the normalised rows the next GEMM reads (post-norm models)
  int ss_parts = 0;
  cg_tensor* ss = nullptr;
  bool logits_gathered = true;   // `logits` holds every rank's slice
  cudaGraphExec_t graph = nullptr;
  int64_t graph_B = -1;
  int64_t graph_gen = -1;        // option generation the graph was captured under
  int64_t step_launches = 0;     // kernels in one decode step
  // all steps of a decode call as one resident kernel (decode_resident.cu), when the model allows
  cg::ResidentPlan* rplan = nullptr;
  int64_t rplan_B = -1, rplan_gen = -1;
  bool resident_off = false;     // this model or device cannot take the resident kernel
  int64_t splitk_floats = 0;
  // decoders built layer by layer (cg_decoder_create_layers): layer list, per-run caches, row tables
  cg::MixedModel* mixed = nullptr;

  int64_t* pos_dev() { return (int64_t*)state->data(); }
  int64_t* count_dev() { return (int64_t*)state->data() + 1; }
};

namespace cg {

// shared by the two layer walks (decoder.cu)
int get_param(cg_decoder* D, const std::string& name, cg_tensor** out, bool required = true);
int norm_weight(cg_decoder* D, const std::string& name, int64_t n, cg_tensor** out, bool required = true);
int set_state(cg_decoder* D, int64_t pos, int64_t generated);

// Decoders built layer by layer (decoder_mixed.cu).  The entry points of decoder.cu call these when
// D->mixed is set.
int mixed_create(cg_decoder* D, const cg_layer_config* layers, int n_layers, const cg_loop_config* loop);
void mixed_destroy(cg_decoder* D);
int mixed_finalize(cg_decoder* D);
int mixed_reset(cg_decoder* D);
// One portion per row: `lens[r]` new tokens of the sequence in slot slots[r], packed row after row in
// `tokens` (device).  want lists packed token places whose logits are asked for, [n_want, vocab] in
// *logits_out.  greedy: every row's last token also goes through the head, and its arg-max becomes
// the row's next token (generated token number 0 of a new record, or the next one).
int mixed_run(cg_decoder* D, const std::vector<int>& slots, const std::vector<int>& lens, const uint32_t* tokens, const int32_t* want,
              int n_want, bool greedy, bool new_record, cg_tensor** logits_out);
// tokens [B, S] as new sequences in slots 0 .. B-1 (fresh) or as the next tokens of the current rows
int mixed_prefill(cg_decoder* D, const cg_tensor* tokens, bool fresh);
int mixed_truncate(cg_decoder* D, int64_t positions);
int mixed_position(cg_decoder* D, int64_t* cached);
// the layers and the head of one decode step for the current rows, tokens taken from D->cur
int mixed_step(cg_decoder* D);
int mixed_begin_decode(cg_decoder* D, int steps);  // checks room and points the row tables at the current rows
void mixed_advance(cg_decoder* D, int steps);

}  // namespace cg
