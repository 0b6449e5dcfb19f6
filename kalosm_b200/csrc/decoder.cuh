// The decoder object behind the C ABI: one struct for every architecture. It owns the session (position, token
// history, greedy and sampled loops, the captured step, logits); the layers are either Llama blocks over
// quantised matrices (llama.cu) or token-mixer layers over dense ones (hybrid.cu).
#pragma once

#include "common.cuh"
#include "fused_step.cuh"
#include "packed_act.cuh"

struct fb200_comm;
struct fb200_hybrid;

struct LayerW {
  fb200_qmatrix *wq = nullptr, *wk = nullptr, *wv = nullptr, *wo = nullptr;
  fb200_qmatrix *gate = nullptr, *up = nullptr, *down = nullptr, *gate_up = nullptr;
  float *attn_norm = nullptr, *ffn_norm = nullptr;
  __half *kc = nullptr, *vc = nullptr;  // [max_batch, Hkv, max_seq, D]
};

struct fb200_llama {
  fb200_device* dev = nullptr;
  fb200_llama_config cfg{};
  fb200_qmatrix *token_embd = nullptr, *output = nullptr;
  float* output_norm = nullptr;
  std::vector<LayerW> layers;
  float *rope_cos = nullptr, *rope_sin = nullptr;
  bool finalized = false;
  // layers made of token mixers (hybrid.cu) instead of `layers`; null for a Llama decoder
  fb200_hybrid* hybrid = nullptr;
  int last_batch = 0, last_seq = 0;  // shape of the last forward pass (fb200_llama_logits_at)
  float* row_logits = nullptr;       // [vocab] one row of fb200_llama_logits_at
  int pos = 0;
  // activation buffers, sized for `rows_cap` rows
  size_t rows_cap = 0;
  float *x = nullptr, *xn = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *att = nullptr,
        *attn_out = nullptr, *hbuf = nullptr, *gbuf = nullptr, *last = nullptr, *logits = nullptr;
  float* att_part = nullptr;
  size_t att_part_bytes = 0;
  uint32_t *ids = nullptr, *next = nullptr, *hist = nullptr;
  int hist_cap = 0;
  // every token fed to or produced by the model since the last reset, [max_batch, max_seq_len + 1]:
  // the penalty window of the samplers
  uint32_t* tok_hist = nullptr;
  float* mu_dev = nullptr;  // [max_batch] Mirostat 2 state of a sampled decode
  int *pos_dev = nullptr, *step_dev = nullptr;
  unsigned long long* argmax_key = nullptr;
  int* att_done = nullptr;  // arrival counters of the attention splits, one per (batch, kv head)
  // single-row step: activation rows travel between kernels in the products' operand form
  fb200_packed_act px, patt, pv, ph;  // residual stream, attention output, attn_out + x, SwiGLU output
  // the same rows (and q / k / v, the residual stream and the attention projection as f32) as flagged
  // rows for the barrier-free variants of the persistent kernel: one slab, zero at creation
  uint8_t* ll_slab = nullptr;
  fb200_ll_act px_ll, patt_ll, pv_ll, ph_ll;
  uint2 *q_ll = nullptr, *k_ll = nullptr, *v_ll = nullptr, *x_ll = nullptr, *attn_ll = nullptr;
  // FB200_FUSED_LL=1 selects the barrier-free variants. Off by default: they are correct (parity
  // tests run both forms) but measured slower so far (2.2 - 2.6 ms per step of the 8B-shaped model
  // against 2.03 ms with grid barriers): the trip a flagged row saves at each phase boundary is
  // outweighed by slower epilogues (8-byte flagged stores), the 86 KB polled row in front of the
  // down projection and a product loop that gets fewer registers.
  bool fused_flagged = false;
  bool fused_is_flagged = false;  // the current program uses the flagged rows
  bool used_key = false;  // the last forward pass left its greedy id in argmax_key, not in next
  // CUDA graph of a single-token step, per batch size
  cudaGraphExec_t graph_exec = nullptr;
  int graph_batch = 0;
  uint64_t graph_kernels = 0;  // kernels inside the captured step
  uint64_t graph_gen = 0;      // the handle's scratch generation the capture recorded addresses of
  // single-sequence step as one persistent kernel: its program (host and device copies)
  bool fused_enabled = true;   // FB200_FUSED=0 keeps the multi-kernel step
  bool fused_valid = false;    // the program matches the current buffers
  bool fused_usable = false;
  std::vector<fb200_fused_phase> prog_host;
  fb200_fused_phase* prog_dev = nullptr;
  // tensor parallelism: cfg holds the local head / ffn counts; the output head has vocab_local rows
  fb200_comm* comm = nullptr;
  int tp_rank = 0, tp_size = 1, vocab_local = 0;
  float* best_val = nullptr;            // [max_batch] value of the local greedy candidate
  unsigned long long* best_pair = nullptr;  // [(1 + size) * max_batch] (value, global id) pairs
};

// Session buffers common to all architectures (llama.cu); the model's dev and cfg are set.
int fb200_decoder_session(fb200_llama* m);

// Token-mixer layers (hybrid.cu). A forward pass takes the ids in m->ids and leaves logits and greedy ids.
int fb200_hybrid_ensure_rows(fb200_llama* m, size_t rows);
int fb200_hybrid_finalize(fb200_llama* m);
int fb200_hybrid_forward(fb200_llama* m, int batch, int seq, bool commit);
int fb200_hybrid_set_tensor(fb200_llama* m, int layer, int which, uint32_t ggml_type, uint64_t n, uint64_t k, const void* bytes_host,
                            size_t nbytes);
int fb200_hybrid_row_logits(fb200_llama* m, size_t row, float* logits_dev);
bool fb200_hybrid_recurrent(const fb200_llama* m);  // some layer carries a state that cannot be rewound
void fb200_hybrid_free(fb200_llama* m);
