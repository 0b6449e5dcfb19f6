// Decoder layers made of token mixers (gated delta rule, latent attention, grouped softmax attention, linear attention)
// over dense weights.
//
// A layer reads its input through one norm, x <- x + m (mixers(h) + ffn(h)), or gives the feed-forward a norm of its own;
// mixers that stand side by side all read h. So all matrices that read the layer's input are stacked into one, w_in =
// [projections of the mixers | gate | up], and those that write the residual are joined along K, w_out = [mixer outputs |
// down]: a layer is
//   product (norms in its prologue for one row; the activation in its epilogue) -> mixers -> product (+ residual).
// Layers inside a loop run several times; every pass has caches and states of its own, and starts with a product over
// [x; embedded x], which is why the residual rows of such a model are 2 hidden wide, the second half holding the embedding.
// One new position of one sequence runs the single-row product with f32 activations; more rows run the tensor-core product
// with bf16 operands, or the f32 product of an F32 model. Steps of one position per sequence are captured
// in a CUDA graph by llama.cu like those of a Llama decoder.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <memory>

#include "decoder.cuh"
#include "dense.cuh"
#include "mixers.cuh"

void fb200_rope_tables_host(int head_dim, int ctx, float theta, float factor, float low_ff, float high_ff, int original_ctx,
                            const float* freq_weight, std::vector<float>& cs, std::vector<float>& sn);
void fb200_rope_tables_yarn_host(int dims, int ctx, double base, double factor, double fast, double slow, double original,
                                 std::vector<float>& cs, std::vector<float>& sn);
int fb200_launch_rms_norm_strided(fb200_device* dev, const float* x, size_t x_stride, const float* res, const float* w, float eps,
                                  size_t rows, size_t n, float* y);
int fb200_launch_argmax(fb200_device* dev, const float* logits, size_t rows, size_t n, uint32_t* ids, float* vals);

namespace {

// One token mixer: an entry of the configuration.
struct Mixer {
  fb200_layer_config c{};
  int layer = 0;                 // the layer it belongs to
  int row0 = 0, rows = 0;        // its projections inside w_in
  int zcol = 0, ko = 0;          // its output inside the operand rows of w_out
  int off_k = 0, off_v = 0, off_g = 0, off_b = 0, off_a = 0, off_dkv = -1;  // relative to row0; q is first
  uint64_t have = 0, need = 0;   // bit per tensor id
  float* bias = nullptr;         // [rows]
  // recurrent kinds: state of one pass and the next one `pass_state` elements further
  int dp = 0, channels = 0;
  float *conv_w = nullptr, *a_log = nullptr, *dt_bias = nullptr, *out_norm = nullptr, *state = nullptr, *ring = nullptr;
  float* decay = nullptr;
  size_t pass_state = 0, pass_ring = 0;
  // attention kinds
  fb200_qmatrix* w_ukv = nullptr;
  int rkp = 0, ldc = 0, vp = 0;
  float *c_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr;
  void* cache = nullptr;
  size_t pass_cache = 0;         // bytes
  float *rope_cos = nullptr, *rope_sin = nullptr;
  bool own_rope = false;
};

struct MixerLayer {
  int first = 0, count = 0;      // its mixers
  int ffn = 0, act = 0, n_plain = 0, ko = 0, passes = 1;
  fb200_qmatrix *w_in = nullptr, *w_out = nullptr;
  float *norm = nullptr, *norm2 = nullptr, *bias = nullptr;
};

struct LayerRun { int layer, pass, enter; };

size_t up_to(size_t n, size_t m) { return (n + m - 1) / m * m; }

}  // namespace

struct fb200_hybrid {
  bool f32 = false;
  fb200_stack_config stack{1.f, 1.f, 0.f, 0, 0, 0};
  std::vector<Mixer> mixers;
  std::vector<MixerLayer> layers;
  std::vector<LayerRun> runs;
  fb200_qmatrix* w_loop = nullptr;
  size_t ldx = 0;           // residual rows
  size_t ldy = 0, ldz = 0;  // widest projection / operand row
  float* x2 = nullptr;      // the other residual buffer of a model with a loop
  float* xend = nullptr;    // where a pass leaves the residual stream
  float *proj = nullptr, *zf = nullptr;
  __nv_bfloat16 *hb = nullptr, *zb = nullptr;
  float *qn = nullptr, *kn = nullptr, *vn = nullptr, *gb = nullptr, *kq = nullptr, *o = nullptr, *seg = nullptr;
  float *qa = nullptr, *part = nullptr;
  int* done = nullptr;      // arrival counters, zero between launches
  size_t done_linear = 0;   // first counter of the linear attention
  __nv_bfloat16* kvx = nullptr;
  size_t kvx_elems = 0;
};

namespace {

// A dense matrix of this model's weight type with zeroed storage, K padded to a multiple of 64.
int make_dense(fb200_device* dev, bool f32, uint64_t n, uint64_t k, fb200_qmatrix** out) {
  auto q = std::unique_ptr<fb200_qmatrix>(new fb200_qmatrix());
  q->dev = dev;
  q->type = q->source_type = f32 ? FB200_F32 : FB200_BF16;
  q->n = n;
  q->k = up_to(k, 64);
  q->data_bytes = q->raw_nbytes = n * q->k * (f32 ? 4 : 2);
  FB_CUDA(dev, cudaMalloc(&q->data, q->data_bytes));
  FB_CUDA(dev, cudaMemsetAsync(q->data, 0, q->data_bytes, dev->stream));
  FB_CUDA(dev, cudaStreamSynchronize(dev->stream));
  *out = q.release();
  return FB200_OK;
}

int alloc_zero(fb200_device* dev, void** p, size_t bytes) {
  FB_CUDA(dev, cudaMalloc(p, bytes ? bytes : 16));
  FB_CUDA(dev, cudaMemset(*p, 0, bytes ? bytes : 16));
  return FB200_OK;
}

float bf16_value(uint16_t u) {
  const uint32_t w = (uint32_t)u << 16;
  float f;
  std::memcpy(&f, &w, 4);
  return f;
}
uint16_t bf16_bits(float f) {  // round to nearest even
  const __nv_bfloat16 h = __float2bfloat16(f);
  uint16_t u;
  std::memcpy(&u, &h, 2);
  return u;
}

// Host bytes of `count` elements (BF16 or F32) as f32
int to_f32(fb200_device* dev, uint32_t type, const void* src, size_t count, std::vector<float>& out) {
  out.resize(count);
  if (type == FB200_F32) std::memcpy(out.data(), src, count * 4);
  else if (type == FB200_BF16)
    for (size_t i = 0; i < count; ++i) out[i] = bf16_value(((const uint16_t*)src)[i]);
  else return fb200_fail(dev, FB200_ERR_UNSUPPORTED_DTYPE, "dense tensors are BF16 or F32, got type %u", type);
  return FB200_OK;
}

// Writes [n, k] host elements into rows row0 .., columns col0 .. of a dense matrix
int put_block(fb200_device* dev, fb200_qmatrix* w, uint64_t row0, uint64_t col0, uint32_t type, uint64_t n, uint64_t k, const void* src) {
  const bool f32 = w->type == FB200_F32;
  const size_t es = f32 ? 4 : 2;
  std::vector<float> wide;
  std::vector<uint16_t> narrow;
  const void* host = src;
  int rc;
  if (type != w->type) {
    if ((rc = to_f32(dev, type, src, n * k, wide))) return rc;
    host = wide.data();
    if (!f32) {
      narrow.resize(n * k);
      for (size_t i = 0; i < narrow.size(); ++i) narrow[i] = bf16_bits(wide[i]);
      host = narrow.data();
    }
  }
  FB_CUDA(dev, cudaMemcpy2D(w->data + (row0 * w->k + col0) * es, w->k * es, host, k * es, k * es, n, cudaMemcpyHostToDevice));
  return FB200_OK;
}

int check_mixer(fb200_device* dev, const fb200_layer_config* all, int i) {
  const auto& c = all[i];
  if (c.ffn < 0 || c.heads <= 0 || c.dim <= 0 || c.vdim <= 0 || (c.ffn_act != FB200_FFN_SWIGLU && c.ffn_act != FB200_FFN_GELU))
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: ffn %d (kind %d) heads %d dim %d vdim %d", i, c.ffn, c.ffn_act, c.heads, c.dim, c.vdim);
  if (c.beside && (i == 0 || c.ffn || c.two_norms))
    return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "entry %d stands beside another mixer: no feed-forward or norm of its own", i);
  if (c.mixer == FB200_MIX_DELTA) {
    if (c.kv_heads <= 0 || c.heads % c.kv_heads || c.conv <= 0 || !fb200_delta_dp(c.dim) || c.vdim > 4096)
      return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: delta rule with %d / %d heads of %d / %d, %d taps", i, c.heads, c.kv_heads,
                        c.dim, c.vdim, c.conv);
  } else if (c.mixer == FB200_MIX_LINEAR) {
    if (!fb200_linear_dp(c.dim) || c.vdim > 4096)
      return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: linear attention with %d heads of %d / %d", i, c.heads, c.dim, c.vdim);
  } else if (c.mixer == FB200_MIX_ATTENTION) {
    if (c.kv_heads <= 0 || c.heads % c.kv_heads || !fb200_attn_covers(c.dim, c.vdim) || c.window < 0 || c.rot_dim < 0 || c.rot_dim % 2 ||
        c.rot_dim > c.dim || c.softcap < 0.f || (c.rot_dim && c.rope_base <= 0.f) || c.yarn_factor < 0.f)
      return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: attention with %d / %d heads of %d / %d, rot_dim %d window %d softcap %g", i, c.heads,
                        c.kv_heads, c.dim, c.vdim, c.rot_dim, c.window, c.softcap);
  } else if (c.mixer == FB200_MIX_LATENT) {
    if (!fb200_latent_covers(c.dim, c.rot_dim, c.vdim, c.kv_rank) || c.window < 0)
      return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: latent attention with dim %d rot_dim %d vdim %d kv_rank %d window %d", i, c.dim,
                        c.rot_dim, c.vdim, c.kv_rank, c.window);
    if (c.kv_from >= 0) {
      if (c.kv_from >= i || all[c.kv_from].mixer != FB200_MIX_LATENT || all[c.kv_from].kv_from >= 0 || all[c.kv_from].kv_rank != c.kv_rank ||
          all[c.kv_from].rot_dim != c.rot_dim || all[c.kv_from].rope_base != c.rope_base)
        return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d: cannot read the latents of layer %d", i, c.kv_from);
    }
  } else {
    return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d: mixer kind %d", i, c.mixer);
  }
  if (c.mixer != FB200_MIX_DELTA && c.mixer != FB200_MIX_LATENT) return FB200_OK;
  if (c.out_scale != 1.f) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d: this mixer's output has no factor", i);
  return FB200_OK;
}

bool same_rope(const fb200_layer_config& a, const fb200_layer_config& b) {
  return a.rot_dim == b.rot_dim && a.rope_base == b.rope_base && (a.mixer == FB200_MIX_ATTENTION) == (b.mixer == FB200_MIX_ATTENTION) &&
         a.yarn_factor == b.yarn_factor && a.yarn_fast == b.yarn_fast && a.yarn_slow == b.yarn_slow && a.yarn_original == b.yarn_original;
}

int make_rope(fb200_llama* m, int i) {
  fb200_device* dev = m->dev;
  auto& all = m->hybrid->mixers;
  Mixer& M = all[i];
  const auto& c = M.c;
  for (int j = 0; j < i && !M.rope_cos; ++j)
    if (all[j].rope_cos && same_rope(all[j].c, c)) { M.rope_cos = all[j].rope_cos; M.rope_sin = all[j].rope_sin; }
  if (M.rope_cos) return FB200_OK;
  std::vector<float> cs, sn;
  if (c.mixer == FB200_MIX_ATTENTION)
    fb200_rope_tables_yarn_host(c.rot_dim, m->cfg.max_seq_len, c.rope_base, c.yarn_factor, c.yarn_fast, c.yarn_slow, c.yarn_original, cs, sn);
  else fb200_rope_tables_host(c.rot_dim, m->cfg.max_seq_len, c.rope_base, 0.f, 1.f, 4.f, m->cfg.max_seq_len, nullptr, cs, sn);
  M.own_rope = true;
  int rc;
  if ((rc = alloc_zero(dev, (void**)&M.rope_cos, cs.size() * 4)) || (rc = alloc_zero(dev, (void**)&M.rope_sin, sn.size() * 4))) return rc;
  FB_CUDA(dev, cudaMemcpy(M.rope_cos, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice));
  FB_CUDA(dev, cudaMemcpy(M.rope_sin, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice));
  return FB200_OK;
}

// Rows of the projections, buffers, caches and states of mixer i; its row0, zcol and layer are set.
int make_mixer(fb200_llama* m, int i, int passes) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  Mixer& M = hy->mixers[i];
  const auto& c = M.c;
  const auto& g = m->cfg;
  auto need = [&](std::initializer_list<int> ids) { for (int t : ids) M.need |= 1ull << t; };
  const size_t es = hy->f32 ? 4 : 2;
  int rc;
  M.ko = c.heads * c.vdim;
  need({FB200_T_MIX_Q, FB200_T_MIX_OUT});
  if (c.mixer == FB200_MIX_DELTA) {
    need({FB200_T_MIX_K, FB200_T_MIX_V, FB200_T_MIX_GATE, FB200_T_MIX_BETA, FB200_T_MIX_DECAY, FB200_T_MIX_Q_CONV, FB200_T_MIX_K_CONV,
          FB200_T_MIX_V_CONV, FB200_T_MIX_A_LOG, FB200_T_MIX_DT_BIAS, FB200_T_MIX_OUT_NORM});
    M.dp = fb200_delta_dp(c.dim);
    M.off_k = c.kv_heads * c.dim;
    M.off_v = 2 * c.kv_heads * c.dim;
    M.channels = M.off_v + c.heads * c.vdim;
    M.off_g = M.channels;
    M.off_b = M.off_g + c.heads * c.vdim;
    M.off_a = M.off_b + c.heads;
    M.rows = M.off_a + c.heads;
    M.pass_state = (size_t)g.max_batch * c.heads * c.vdim * M.dp;
    M.pass_ring = (size_t)g.max_batch * c.conv * M.channels;
    if ((rc = alloc_zero(dev, (void**)&M.conv_w, (size_t)M.channels * c.conv * 4)) || (rc = alloc_zero(dev, (void**)&M.a_log, c.heads * 4)) ||
        (rc = alloc_zero(dev, (void**)&M.dt_bias, c.heads * 4)) || (rc = alloc_zero(dev, (void**)&M.out_norm, c.vdim * 4)) ||
        (rc = alloc_zero(dev, (void**)&M.ring, passes * M.pass_ring * 4)))
      return rc;
  } else if (c.mixer == FB200_MIX_LINEAR) {
    need({FB200_T_MIX_K, FB200_T_MIX_V, FB200_T_MIX_GATE, FB200_T_MIX_OUT_NORM, FB200_T_MIX_HEAD_DECAY});
    M.dp = fb200_linear_dp(c.dim);
    M.off_k = c.heads * c.dim;
    M.off_v = 2 * M.off_k;
    M.off_g = M.off_v + M.ko;
    M.rows = M.off_g + M.ko;
    M.pass_state = (size_t)g.max_batch * c.heads * c.vdim * M.dp;
    if ((rc = alloc_zero(dev, (void**)&M.out_norm, (size_t)M.ko * 4)) ||
        (rc = alloc_zero(dev, (void**)&M.decay, (size_t)c.heads * (FB200_LINEAR_CHUNK + 1) * 4)))
      return rc;
  } else if (c.mixer == FB200_MIX_ATTENTION) {
    need({FB200_T_MIX_K, FB200_T_MIX_V});
    M.off_k = c.heads * c.dim;
    M.off_v = M.off_k + c.kv_heads * c.dim;
    M.rows = M.off_v + c.kv_heads * c.vdim;
    if (c.parts & FB200_ATTN_GATE) {
      need({FB200_T_MIX_GATE});
      M.off_g = M.rows;
      M.rows += c.heads;
    }
    if (c.parts & FB200_ATTN_BIAS) need({FB200_T_MIX_Q_BIAS, FB200_T_MIX_K_BIAS, FB200_T_MIX_V_BIAS});
    if (c.parts & FB200_ATTN_QK_NORM) {
      need({FB200_T_MIX_Q_NORM, FB200_T_MIX_K_NORM});
      if ((rc = alloc_zero(dev, (void**)&M.q_norm, c.dim * 4)) || (rc = alloc_zero(dev, (void**)&M.k_norm, c.dim * 4))) return rc;
    }
    if (c.parts & FB200_ATTN_SINK) {
      need({FB200_T_MIX_SINK});
      if ((rc = alloc_zero(dev, (void**)&M.sink, c.heads * 4))) return rc;
    }
    M.dp = (int)up_to(c.dim, 8);
    M.vp = (int)up_to(c.vdim, 8);
    M.ldc = c.kv_heads * (M.dp + M.vp);
    M.pass_cache = (size_t)g.max_batch * g.max_seq_len * M.ldc * es;
    if (c.rot_dim && (rc = make_rope(m, i))) return rc;
  } else {
    need({FB200_T_MIX_GATE, FB200_T_MIX_UK, FB200_T_MIX_UV});
    M.rkp = (int)up_to(c.kv_rank, 64);
    M.ldc = (int)up_to(c.kv_rank + c.rot_dim, 8);
    M.off_g = c.heads * (c.dim + c.rot_dim);
    M.rows = M.off_g + c.heads;
    if ((rc = make_dense(dev, hy->f32, (uint64_t)c.heads * (c.dim + c.vdim), c.kv_rank, &M.w_ukv))) return rc;
    if (c.kv_from >= 0) {
      if (hy->layers[hy->mixers[c.kv_from].layer].passes != passes)
        return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "entry %d: the latents of entry %d belong to another loop", i, c.kv_from);
      M.cache = hy->mixers[c.kv_from].cache;
    } else {
      need({FB200_T_MIX_DKV, FB200_T_MIX_DKV_NORM});
      M.off_dkv = M.rows;
      M.rows += c.kv_rank + c.rot_dim;
      if ((rc = alloc_zero(dev, (void**)&M.c_norm, c.kv_rank * 4))) return rc;
    }
    M.pass_cache = (size_t)g.max_batch * g.max_seq_len * M.ldc * es;
    if ((rc = make_rope(m, i))) return rc;
  }
  if (M.pass_state && (rc = alloc_zero(dev, (void**)&M.state, passes * M.pass_state * 4))) return rc;
  if (M.pass_cache && !M.cache && (rc = alloc_zero(dev, &M.cache, passes * M.pass_cache))) return rc;
  return FB200_OK;
}

int make_layer(fb200_llama* m, int li) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  MixerLayer& L = hy->layers[li];
  Mixer& head = hy->mixers[L.first];
  const size_t E = m->cfg.hidden;
  int rc;
  L.ffn = head.c.ffn;
  L.act = head.c.ffn_act;
  head.need |= 1ull << FB200_T_ATTN_NORM;
  if (L.ffn) {
    head.need |= 1ull << FB200_T_FFN_UP | 1ull << FB200_T_FFN_DOWN;
    if (L.act == FB200_FFN_SWIGLU) head.need |= 1ull << FB200_T_FFN_GATE;
    if (head.c.two_norms) {
      head.need |= 1ull << FB200_T_FFN_NORM;
      if ((rc = alloc_zero(dev, (void**)&L.norm2, E * 4))) return rc;
    }
  }
  bool bias = false;
  for (int k = 0; k < L.count; ++k) {
    Mixer& M = hy->mixers[L.first + k];
    M.layer = li;
    M.row0 = (int)up_to(L.n_plain, 8);  // rows in between stay zero
    M.zcol = L.ko;
    if ((rc = make_mixer(m, L.first + k, L.passes))) return rc;
    L.n_plain = M.row0 + M.rows;
    L.ko += M.ko;
    bias = bias || (M.c.mixer == FB200_MIX_ATTENTION && (M.c.parts & FB200_ATTN_BIAS));
  }
  if (bias) {
    if ((rc = alloc_zero(dev, (void**)&L.bias, (size_t)L.n_plain * 4))) return rc;
    for (int k = 0; k < L.count; ++k) hy->mixers[L.first + k].bias = L.bias + hy->mixers[L.first + k].row0;
  }
  const int ffr = L.act == FB200_FFN_SWIGLU ? 2 * L.ffn : L.ffn;
  if ((rc = make_dense(dev, hy->f32, (uint64_t)L.n_plain + ffr, E, &L.w_in)) || (rc = make_dense(dev, hy->f32, E, (uint64_t)L.ko + L.ffn, &L.w_out)) ||
      (rc = alloc_zero(dev, (void**)&L.norm, E * 4)))
    return rc;
  hy->ldy = std::max(hy->ldy, up_to(L.n_plain, 8));
  hy->ldz = std::max(hy->ldz, up_to(L.ko + L.ffn, 8));
  return FB200_OK;
}

// A prompt pass long enough for the expansion of keys and values to pay (tensor-core attention over them)
bool expanded(const fb200_hybrid* hy, const Mixer& M, int seq) {
  const auto& c = M.c;
  return !hy->f32 && seq >= 16 && M.zcol % 8 == 0 && fb200_latent_prefill_covers(c.heads, c.dim, c.rot_dim, c.vdim, c.kv_rank, c.scale);
}
// The same for grouped attention (tensor-core kernel against the row-by-row one)
bool attn_tiled(const fb200_hybrid* hy, const Mixer& M, int seq) {
  return !hy->f32 && seq >= 16 && fb200_attn_prefill_covers(M.c.heads, M.c.dim, M.c.vdim, M.c.scale);
}

// y: the mixer's projections, z: its columns of the operand rows
int run_mixer(fb200_llama* m, const Mixer& M, int pass, int batch, int seq, bool commit, const float* y, void* z, bool wide) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const auto& c = M.c;
  const int rows = batch * seq;
  int rc;
  if (c.mixer == FB200_MIX_DELTA) {
    fb200_delta_args a = {};
    a.y = y; a.ldy = hy->ldy; a.off_v = M.off_v; a.off_g = M.off_g; a.off_b = M.off_b; a.off_a = M.off_a;
    a.conv_w = M.conv_w; a.a_log = M.a_log; a.dt_bias = M.dt_bias; a.out_norm = M.out_norm; a.eps = m->cfg.rms_eps;
    a.state = M.state + pass * M.pass_state; a.ring = M.ring + pass * M.pass_ring; a.b = batch; a.s = seq; a.h = c.heads; a.hk = c.kv_heads;
    a.d = c.dim; a.v = c.vdim; a.dp = M.dp; a.taps = c.conv; a.channels = M.channels; a.pos_dev = m->pos_dev; a.z = z; a.ldz = hy->ldz;
    a.z_bf16 = !wide; a.commit = commit;
    a.qn = hy->qn; a.kn = hy->kn; a.vn = hy->vn; a.gb = hy->gb; a.kq = hy->kq; a.o = hy->o;
    return seq == 1 ? fb200_delta_step(dev, a) : fb200_delta_prompt(dev, a);
  }
  if (c.mixer == FB200_MIX_LINEAR) {
    fb200_linear_args a = {};
    a.y = y; a.ldy = hy->ldy; a.off_k = M.off_k; a.off_v = M.off_v; a.off_g = M.off_g; a.decay = M.decay; a.out_norm = M.out_norm;
    a.eps = m->cfg.rms_eps; a.out_scale = c.out_scale; a.state = M.state + pass * M.pass_state; a.b = batch; a.s = seq; a.h = c.heads;
    a.d = c.dim; a.v = c.vdim; a.dp = M.dp; a.pos_dev = m->pos_dev; a.z = z; a.ldz = hy->ldz; a.z_bf16 = !wide; a.commit = commit;
    a.o = hy->o; a.done = hy->done + hy->done_linear; a.bf16 = !hy->f32;
    a.q16 = (__nv_bfloat16*)hy->qn; a.k16 = (__nv_bfloat16*)hy->kn; a.v16 = (__nv_bfloat16*)hy->vn;
    a.seg = hy->seg;
    return seq == 1 ? fb200_linear_step(dev, a) : fb200_linear_prompt(dev, a);
  }
  if (c.mixer == FB200_MIX_ATTENTION) {
    fb200_attn_args a = {};
    a.y = y; a.ldy = hy->ldy; a.off_k = M.off_k; a.off_v = M.off_v; a.off_g = c.parts & FB200_ATTN_GATE ? M.off_g : -1;
    a.q_norm = M.q_norm; a.k_norm = M.k_norm; a.sink = M.sink; a.eps = m->cfg.rms_eps; a.scale = c.scale; a.softcap = c.softcap;
    a.out_scale = c.out_scale; a.window = c.window; a.rope_cos = M.rope_cos; a.rope_sin = M.rope_sin; a.r = c.rot_dim;
    a.cache = (uint8_t*)M.cache + pass * M.pass_cache; a.cache_f32 = hy->f32; a.ldc = M.ldc; a.cap = m->cfg.max_seq_len;
    a.b = batch; a.s = seq; a.h = c.heads; a.g = c.kv_heads; a.d = c.dim; a.v = c.vdim; a.dp = M.dp; a.vp = M.vp;
    a.pos_dev = m->pos_dev; a.pos = m->pos; a.z = z; a.ldz = hy->ldz; a.z_bf16 = !wide; a.qn = hy->qn; a.part = hy->part; a.done = hy->done;
    return attn_tiled(hy, M, seq) ? fb200_attn_prefill(dev, a) : fb200_attn_rows(dev, a);
  }
  fb200_latent_args a = {};
  a.y = y; a.ldy = hy->ldy; a.off_g = M.off_g; a.off_dkv = M.off_dkv; a.w_ukv = M.w_ukv->data; a.c_norm = M.c_norm;
  a.eps = m->cfg.rms_eps; a.cache = (uint8_t*)M.cache + pass * M.pass_cache; a.cache_f32 = hy->f32; a.ldc = M.ldc; a.cap = m->cfg.max_seq_len;
  a.rope_cos = M.rope_cos; a.rope_sin = M.rope_sin; a.b = batch; a.s = seq; a.h = c.heads; a.d = c.dim; a.r = c.rot_dim; a.v = c.vdim;
  a.rk = c.kv_rank; a.rkp = M.rkp; a.window = c.window; a.scale = c.scale; a.pos_dev = m->pos_dev; a.pos = m->pos;
  a.z = z; a.ldz = hy->ldz; a.z_bf16 = !wide; a.qa = hy->qa; a.part = hy->part;
  if (expanded(hy, M, seq)) {
    a.kvx = hy->kvx;
    if ((rc = fb200_latent_append(dev, a))) return rc;
    return fb200_latent_prefill(dev, a, M.w_ukv);
  }
  a.nsplit = fb200_latent_nsplit(dev, rows, c.heads, c.window, m->cfg.max_seq_len);
  return fb200_latent_rows(dev, a);
}

// x: the residual rows, updated in place
int run_layer(fb200_llama* m, const MixerLayer& L, int pass, float* x, int batch, int seq, bool commit) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const int rows = batch * seq, E = m->cfg.hidden;
  const bool wide = hy->f32 || rows == 1;  // f32 operand rows
  const float eps = m->cfg.rms_eps;
  int rc;
  fb200_dense_job in;
  in.w = L.w_in; in.m = rows; in.kx = E;
  if (rows == 1) {
    in.x = x; in.ldx = E; in.norm_w = L.norm; in.ff_norm_w = L.norm2; in.eps = eps;
  } else if (hy->f32) {
    if ((rc = fb200_launch_rms_norm_strided(dev, x, hy->ldx, nullptr, L.norm, eps, rows, E, m->xn))) return rc;
    in.x = m->xn; in.ldx = E;
    if (L.norm2) {
      in.ff_off = (size_t)rows * E;
      if ((rc = fb200_launch_rms_norm_strided(dev, x, hy->ldx, nullptr, L.norm2, eps, rows, E, m->xn + in.ff_off))) return rc;
    }
  } else {
    const int np = (int)L.w_in->k;
    if ((rc = fb200_rows_to_bf16(dev, x, hy->ldx, L.norm, L.norm2, eps, rows, E, np, hy->hb))) return rc;
    in.x = hy->hb; in.ldx = L.norm2 ? 2 * np : np; in.ff_off = L.norm2 ? np : 0;
  }
  in.n_plain = L.n_plain; in.bias = L.bias; in.y = hy->proj; in.ldy = hy->ldy;
  in.act = L.act; in.ff = L.ffn; in.gate0 = L.n_plain; in.up0 = L.n_plain + (L.act == FB200_FFN_SWIGLU ? L.ffn : 0);
  in.z = wide ? (void*)(hy->zf + L.ko) : (void*)(hy->zb + L.ko); in.ldz = hy->ldz;
  if ((rc = fb200_dense_product(dev, in))) return rc;

  for (int k = 0; k < L.count; ++k) {
    const Mixer& M = hy->mixers[L.first + k];
    void* z = wide ? (void*)(hy->zf + M.zcol) : (void*)(hy->zb + M.zcol);
    if ((rc = run_mixer(m, M, pass, batch, seq, commit, hy->proj + M.row0, z, wide))) return rc;
  }

  fb200_dense_job out;
  out.w = L.w_out; out.m = rows; out.x = wide ? (void*)hy->zf : (void*)hy->zb; out.ldx = hy->ldz; out.kx = L.ko + L.ffn;
  out.n_plain = E; out.y = x; out.ldy = hy->ldx; out.add = x; out.ldadd = hy->ldx; out.alpha = hy->stack.residual_mult;
  return fb200_dense_product(dev, out);
}

// In front of a pass of the loop: the x half of `to` = W_loop [x; embedded x]. Rows of both are [x | embedded x].
int enter_pass(fb200_llama* m, const float* from, float* to, int rows) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const int E = m->cfg.hidden;
  fb200_dense_job j;
  j.w = hy->w_loop; j.m = rows; j.kx = 2 * E; j.n_plain = E; j.y = to; j.ldy = hy->ldx;
  if (hy->f32 || rows == 1) {
    j.x = from; j.ldx = hy->ldx;
  } else {
    const int np = (int)hy->w_loop->k;
    const int rc = fb200_rows_to_bf16(dev, from, hy->ldx, nullptr, nullptr, 0.f, rows, 2 * E, np, hy->hb);
    if (rc) return rc;
    j.x = hy->hb; j.ldx = np;
  }
  return fb200_dense_product(dev, j);
}

// Residual rows from the embedding table (dense row-major bf16 or f32): x, and in a model with a loop the second half of
// the rows of both buffers.
template <typename T>
__global__ void __launch_bounds__(256)
embed_rows_kernel(const T* __restrict__ table, const uint32_t* __restrict__ ids, uint32_t vocab, int n, float scale, float* x, float* x2, size_t ldx) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const size_t row = blockIdx.x;
  const uint32_t id = ids[row];
  for (int i = threadIdx.x; i < n; i += 256) {
    const float v = id < vocab ? (float)table[(size_t)id * n + i] * scale : 0.f;
    x[row * ldx + i] = v;
    if (x2) {
      x[row * ldx + n + i] = v;
      x2[row * ldx + n + i] = v;
    }
  }
}

}  // namespace

int fb200_hybrid_ensure_rows(fb200_llama* m, size_t rows) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const size_t E = m->cfg.hidden, nb = m->cfg.max_batch;
  size_t q = 0, qk = 0, hv = 0, o = 0, heads = 0, kvh = 0, qa = 0, part = 0, done = 0, seg = 0;
  for (const auto& M : hy->mixers) {
    const auto& c = M.c;
    if (c.mixer == FB200_MIX_DELTA) {
      qk = std::max(qk, (size_t)c.kv_heads * M.dp);
      hv = std::max(hv, (size_t)M.ko);
      heads = std::max(heads, (size_t)c.heads);
      kvh = std::max(kvh, (size_t)c.kv_heads);
    } else if (c.mixer == FB200_MIX_LINEAR) {
      o = std::max(o, (size_t)M.ko);
      if (!hy->f32) {
        qk = std::max(qk, (size_t)c.heads * M.dp / 2);
        hv = std::max(hv, c.heads * up_to(c.vdim, 8) / 2);
        seg = std::max(seg, FB200_LINEAR_SEGMENTS * M.pass_state);
      }
    } else if (c.mixer == FB200_MIX_ATTENTION) {
      q = std::max(q, (size_t)c.heads * M.dp);
      part = std::max(part, fb200_attn_part_floats(dev, c.vdim));
      done = std::max(done, rows * (size_t)c.heads);
    } else {
      // rows of the latent-space path: all of them, or fewer where longer passes expand keys and values
      const bool exp = expanded(hy, M, 16);
      const size_t r = exp ? std::min(rows, (size_t)16 * nb) : rows;
      qa = std::max(qa, r * c.heads * (size_t)(c.kv_rank + c.rot_dim));
      part = std::max(part, std::max(r * c.heads, (size_t)8 * dev->sm_count) * (size_t)(c.kv_rank + 2));
    }
  }
  q = std::max(q, qk);
  for (const auto& M : hy->mixers)
    if (M.c.mixer == FB200_MIX_DELTA) o = std::max(o, hv);
  hy->done_linear = done;
  bool norm2 = false;
  for (const auto& L : hy->layers) norm2 = norm2 || L.norm2;
  const size_t hb = std::max((norm2 ? 2 : 1) * up_to(E, 64), hy->w_loop ? (size_t)hy->w_loop->k : 0);
  struct { void** p; size_t bytes; } bufs[] = {
      {(void**)&m->x, rows * hy->ldx * 4}, {(void**)&hy->x2, hy->w_loop ? rows * hy->ldx * 4 : 0}, {(void**)&m->xn, (norm2 ? 2 : 1) * rows * E * 4},
      {(void**)&hy->proj, rows * hy->ldy * 4}, {(void**)&hy->zf, rows * hy->ldz * 4}, {(void**)&hy->hb, rows * hb * 2},
      {(void**)&hy->zb, rows * hy->ldz * 2}, {(void**)&hy->qn, rows * q * 4}, {(void**)&hy->kn, rows * qk * 4}, {(void**)&hy->vn, rows * hv * 4},
      {(void**)&hy->gb, rows * heads * 8}, {(void**)&hy->kq, (rows + 3 * nb) / 4 * kvh * 64 + 64}, {(void**)&hy->o, rows * o * 4}, {(void**)&hy->seg, seg * 4},
      {(void**)&hy->qa, qa * 4}, {(void**)&hy->part, part * 4}, {(void**)&hy->done, (done + nb) * 4}};
  for (auto& b : bufs) {
    if (*b.p) { cudaFree(*b.p); *b.p = nullptr; }
    FB_CUDA(dev, cudaMalloc(b.p, b.bytes ? b.bytes : 16));
    if (dev->poison) FB_CUDA(dev, cudaMemsetAsync(*b.p, 0xFF, b.bytes ? b.bytes : 16, dev->stream));
  }
  FB_CUDA(dev, cudaMemsetAsync(hy->done, 0, (done + nb) * 4, dev->stream));
  hy->xend = m->x;
  return FB200_OK;
}

int fb200_hybrid_finalize(fb200_llama* m) {
  fb200_hybrid* hy = m->hybrid;
  if (!m->output) return fb200_fail(m->dev, FB200_ERR_INVALID_ARGUMENT, "the output head is not set");
  if (hy->stack.loop_times && !hy->w_loop) return fb200_fail(m->dev, FB200_ERR_INVALID_ARGUMENT, "the loop's input matrix is not set");
  for (size_t i = 0; i < hy->mixers.size(); ++i) {
    const Mixer& M = hy->mixers[i];
    if ((M.have & M.need) != M.need)
      return fb200_fail(m->dev, FB200_ERR_INVALID_ARGUMENT, "layer %zu is missing tensors (ids 0x%llx)", i, (unsigned long long)(M.need & ~M.have));
  }
  return FB200_OK;
}

int fb200_hybrid_row_logits(fb200_llama* m, size_t row, float* logits_dev) {
  fb200_dense_job j;
  j.w = m->output; j.m = 1; j.x = m->hybrid->xend + row * m->hybrid->ldx; j.ldx = m->cfg.hidden; j.kx = m->cfg.hidden;
  j.norm_w = m->output_norm; j.eps = m->cfg.rms_eps; j.n_plain = m->cfg.vocab; j.y = logits_dev; j.ldy = m->cfg.vocab;
  j.softcap = m->hybrid->stack.logit_softcap;
  return fb200_dense_product(m->dev, j);
}

int fb200_hybrid_forward(fb200_llama* m, int batch, int seq, bool commit) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  int rc;
  size_t kvx = 0;
  for (const auto& M : hy->mixers)
    if (M.c.mixer == FB200_MIX_LATENT && expanded(hy, M, seq)) {
      const int before = M.c.window && M.c.window - 1 < m->pos ? M.c.window - 1 : m->pos;
      kvx = std::max(kvx, (size_t)batch * (before + seq) * M.c.heads * (M.c.dim + M.c.vdim));
    }
  if (kvx > hy->kvx_elems) {
    FB_CUDA(dev, cudaStreamSynchronize(dev->stream));
    if (hy->kvx) cudaFree(hy->kvx);
    hy->kvx = nullptr;
    hy->kvx_elems = 0;
    FB_CUDA(dev, cudaMalloc(&hy->kvx, kvx * 2));
    hy->kvx_elems = kvx;
  }
  const int E = m->cfg.hidden, rows = batch * seq;
  float *x = m->x, *other = hy->w_loop ? hy->x2 : nullptr;
  const auto& emb = *m->token_embd;
  if (emb.type == FB200_F32)
    rc = fb200_launch(dev, embed_rows_kernel<float>, dim3((unsigned)rows), dim3(256), 0, false, (const float*)emb.data, m->ids, (uint32_t)m->cfg.vocab,
                      E, hy->stack.embed_scale, x, other, hy->ldx);
  else
    rc = fb200_launch(dev, embed_rows_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(256), 0, false, (const __nv_bfloat16*)emb.data, m->ids,
                      (uint32_t)m->cfg.vocab, E, hy->stack.embed_scale, x, other, hy->ldx);
  if (rc) return rc;
  for (const LayerRun& r : hy->runs) {
    if (r.enter) {
      if ((rc = enter_pass(m, x, other, rows))) return rc;
      std::swap(x, other);
    }
    if ((rc = run_layer(m, hy->layers[r.layer], r.pass, x, batch, seq, commit))) return rc;
  }
  hy->xend = x;
  // final norm and output head on the last position of every sequence
  if (batch == 1) {
    if ((rc = fb200_hybrid_row_logits(m, (size_t)seq - 1, m->logits))) return rc;
  } else {
    fb200_dense_job j;
    j.w = m->output; j.m = batch; j.kx = E; j.n_plain = m->cfg.vocab; j.y = m->logits; j.ldy = m->cfg.vocab; j.softcap = hy->stack.logit_softcap;
    const float* last = x + (size_t)(seq - 1) * hy->ldx;
    if (hy->f32) {
      if ((rc = fb200_launch_rms_norm_strided(dev, last, (size_t)seq * hy->ldx, nullptr, m->output_norm, m->cfg.rms_eps, batch, E, m->last))) return rc;
      j.x = m->last; j.ldx = E;
    } else {
      if ((rc = fb200_rows_to_bf16(dev, last, (size_t)seq * hy->ldx, m->output_norm, nullptr, m->cfg.rms_eps, batch, E, (int)m->output->k, hy->hb))) return rc;
      j.x = hy->hb; j.ldx = m->output->k;
    }
    if ((rc = fb200_dense_product(dev, j))) return rc;
  }
  return fb200_launch_argmax(dev, m->logits, batch, m->cfg.vocab, m->next, nullptr);
}

bool fb200_hybrid_recurrent(const fb200_llama* m) {
  if (!m->hybrid) return false;
  for (const auto& M : m->hybrid->mixers)
    if (M.c.mixer == FB200_MIX_DELTA || M.c.mixer == FB200_MIX_LINEAR) return true;
  return false;
}

void fb200_hybrid_free(fb200_llama* m) {
  fb200_hybrid* hy = m->hybrid;
  if (!hy) return;
  for (auto& M : hy->mixers) {
    if (M.w_ukv) fb200_qmatrix_free(M.w_ukv);
    void* bufs[] = {M.conv_w, M.a_log, M.dt_bias, M.out_norm, M.state, M.ring, M.decay, M.c_norm, M.q_norm, M.k_norm, M.sink,
                    M.c.mixer == FB200_MIX_LATENT && M.c.kv_from >= 0 ? nullptr : M.cache, M.own_rope ? M.rope_cos : nullptr, M.own_rope ? M.rope_sin : nullptr};
    for (void* b : bufs) if (b) cudaFree(b);
  }
  for (auto& L : hy->layers) {
    for (fb200_qmatrix* q : {L.w_in, L.w_out})
      if (q) fb200_qmatrix_free(q);
    void* bufs[] = {L.norm, L.norm2, L.bias};
    for (void* b : bufs) if (b) cudaFree(b);
  }
  if (hy->w_loop) fb200_qmatrix_free(hy->w_loop);
  void* bufs[] = {hy->proj, hy->zf, hy->hb, hy->zb, hy->qn, hy->kn, hy->vn, hy->gb, hy->kq, hy->o, hy->seg, hy->qa, hy->part, hy->done, hy->x2, hy->kvx};
  for (void* b : bufs) if (b) cudaFree(b);
  delete hy;
  m->hybrid = nullptr;
}

int fb200_hybrid_set_tensor(fb200_llama* m, int layer, int which, uint32_t type, uint64_t n, uint64_t k, const void* src, size_t nbytes) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const uint64_t E = m->cfg.hidden, vocab = m->cfg.vocab;
  if (type != FB200_BF16 && type != FB200_F32)
    return fb200_fail(dev, FB200_ERR_UNSUPPORTED_DTYPE, "token-mixer layers take BF16 or F32 tensors, got type %u", type);
  if (!k) k = 1;
  if (!src || nbytes != n * k * (type == FB200_F32 ? 4 : 2))
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "tensor %d: %zu bytes for [%llu, %llu]", which, nbytes, (unsigned long long)n, (unsigned long long)k);
  uint64_t en = 0, ek = 1;
  auto shape_ok = [&]() {
    if (n == en && k == ek) return (int)FB200_OK;
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d tensor %d has shape [%llu, %llu], expected [%llu, %llu]", layer, which,
                      (unsigned long long)n, (unsigned long long)k, (unsigned long long)en, (unsigned long long)ek);
  };
  int rc;
  auto vec = [&](float* dst) -> int {
    std::vector<float> f;
    if ((rc = to_f32(dev, type, src, n * k, f))) return rc;
    FB_CUDA(dev, cudaMemcpy(dst, f.data(), f.size() * 4, cudaMemcpyHostToDevice));
    return FB200_OK;
  };
  if (which == FB200_T_TOKEN_EMBD || which == FB200_T_OUTPUT) {
    en = vocab; ek = E;
    if ((rc = shape_ok())) return rc;
    if (which == FB200_T_TOKEN_EMBD) {
      if (m->token_embd) { fb200_qmatrix_free(m->token_embd); m->token_embd = nullptr; }
      const uint64_t shape[2] = {n, k};
      return fb200_qmatrix_from_raw_bytes(dev, shape, 2, src, nbytes, type, &m->token_embd);
    }
    if (!m->output && (rc = make_dense(dev, hy->f32, vocab, E, &m->output))) return rc;
    return put_block(dev, m->output, 0, 0, type, n, k, src);
  }
  if (which == FB200_T_OUTPUT_NORM) {
    en = E;
    if ((rc = shape_ok())) return rc;
    if (!m->output_norm) FB_CUDA(dev, cudaMalloc(&m->output_norm, E * 4));
    return vec(m->output_norm);
  }
  if (which == FB200_T_LOOP_IN) {
    if (!hy->stack.loop_times) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "the model has no loop");
    en = E; ek = 2 * E;
    if ((rc = shape_ok())) return rc;
    if (!hy->w_loop && (rc = make_dense(dev, hy->f32, en, ek, &hy->w_loop))) return rc;
    return put_block(dev, hy->w_loop, 0, 0, type, n, k, src);
  }
  if (layer < 0 || layer >= (int)hy->mixers.size() || which < 0 || which > 63) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d tensor %d", layer, which);
  Mixer& M = hy->mixers[layer];
  MixerLayer& L = hy->layers[M.layer];
  const auto& c = M.c;
  if (!(M.need >> which & 1ull)) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d has no tensor %d", layer, which);
  const bool latent = c.mixer == FB200_MIX_LATENT, linear = c.mixer == FB200_MIX_LINEAR, attn = c.mixer == FB200_MIX_ATTENTION;
  // rows of q, of k, of v, of the gate
  const uint64_t hv = (uint64_t)c.heads * c.vdim, qr = (uint64_t)(c.mixer == FB200_MIX_DELTA ? c.kv_heads : c.heads) * (c.dim + (latent ? c.rot_dim : 0)),
                 kr = linear ? qr : (uint64_t)c.kv_heads * c.dim, vr = attn ? (uint64_t)c.kv_heads * c.vdim : hv, gr = latent || attn ? c.heads : hv;
  const uint64_t ffr = (uint64_t)L.n_plain + (L.act == FB200_FFN_SWIGLU ? L.ffn : 0);
  fb200_qmatrix* w = L.w_in;
  float* vd = nullptr;
  bool conv = false;
  uint64_t row0 = 0, col0 = 0;
  ek = E;
  auto vector = [&](uint64_t len, float* dst) { en = len; ek = 1; vd = dst; };
  auto rows = [&](uint64_t len, int off) { en = len; row0 = (uint64_t)M.row0 + off; };
  switch (which) {
    case FB200_T_ATTN_NORM: vector(E, L.norm); break;
    case FB200_T_FFN_NORM: vector(E, L.norm2); break;
    case FB200_T_FFN_GATE: en = L.ffn; row0 = L.n_plain; break;
    case FB200_T_FFN_UP: en = L.ffn; row0 = ffr; break;
    case FB200_T_FFN_DOWN: en = E; ek = L.ffn; w = L.w_out; col0 = L.ko; break;
    case FB200_T_MIX_OUT: en = E; ek = hv; w = L.w_out; col0 = M.zcol; break;
    case FB200_T_MIX_Q: rows(qr, 0); break;
    case FB200_T_MIX_K: rows(kr, M.off_k); break;
    case FB200_T_MIX_V: rows(vr, M.off_v); break;
    case FB200_T_MIX_GATE: rows(gr, M.off_g); break;
    case FB200_T_MIX_BETA: rows(c.heads, M.off_b); break;
    case FB200_T_MIX_DECAY: rows(c.heads, M.off_a); break;
    case FB200_T_MIX_DKV: rows((uint64_t)c.kv_rank + c.rot_dim, M.off_dkv); break;
    case FB200_T_MIX_UK: en = (uint64_t)c.heads * c.dim; ek = c.kv_rank; w = M.w_ukv; break;
    case FB200_T_MIX_UV: en = hv; ek = c.kv_rank; w = M.w_ukv; row0 = (uint64_t)c.heads * c.dim; break;
    case FB200_T_MIX_Q_CONV: en = qr; ek = c.conv; conv = true; break;
    case FB200_T_MIX_K_CONV: en = kr; ek = c.conv; col0 = qr; conv = true; break;
    case FB200_T_MIX_V_CONV: en = hv; ek = c.conv; col0 = qr + kr; conv = true; break;
    case FB200_T_MIX_A_LOG: vector(c.heads, M.a_log); break;
    case FB200_T_MIX_DT_BIAS: vector(c.heads, M.dt_bias); break;
    case FB200_T_MIX_OUT_NORM: vector(linear ? hv : c.vdim, M.out_norm); break;
    case FB200_T_MIX_DKV_NORM: vector(c.kv_rank, M.c_norm); break;
    case FB200_T_MIX_Q_NORM: vector(c.dim, M.q_norm); break;
    case FB200_T_MIX_K_NORM: vector(c.dim, M.k_norm); break;
    case FB200_T_MIX_SINK: vector(c.heads, M.sink); break;
    case FB200_T_MIX_Q_BIAS: vector(qr, M.bias); break;
    case FB200_T_MIX_K_BIAS: vector(kr, M.bias + M.off_k); break;
    case FB200_T_MIX_V_BIAS: vector(vr, M.bias + M.off_v); break;
    case FB200_T_MIX_HEAD_DECAY: vector(c.heads, M.decay); break;
    default: return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "tensor id %d", which);
  }
  if ((rc = shape_ok())) return rc;
  if (conv) {  // convolution taps [channels, taps] -> columns col0 .. of [taps][channels]
    std::vector<float> f;
    if ((rc = to_f32(dev, type, src, n * k, f))) return rc;
    std::vector<float> t(f.size());
    for (uint64_t i = 0; i < n; ++i)
      for (uint64_t j = 0; j < k; ++j) t[j * n + i] = f[i * k + j];
    FB_CUDA(dev, cudaMemcpy2D(M.conv_w + col0, (size_t)M.channels * 4, t.data(), n * 4, n * 4, k, cudaMemcpyHostToDevice));
    M.have |= 1ull << which;
    return FB200_OK;
  }
  if (which == FB200_T_MIX_HEAD_DECAY) {  // powers 0 .. chunk of every head's decay
    std::vector<float> f;
    if ((rc = to_f32(dev, type, src, n * k, f))) return rc;
    std::vector<float> t;
    for (float d : f)
      for (int e = 0; e <= FB200_LINEAR_CHUNK; ++e) t.push_back((float)std::pow((double)d, e));
    FB_CUDA(dev, cudaMemcpy(M.decay, t.data(), t.size() * 4, cudaMemcpyHostToDevice));
    M.have |= 1ull << which;
    return FB200_OK;
  }
  rc = vd ? vec(vd) : put_block(dev, w, row0, col0, type, n, k, src);
  if (!rc) M.have |= 1ull << which;
  return rc;
}

extern "C" int fb200_llama_create_layers(fb200_device* dev, const fb200_llama_config* cfg, const fb200_layer_config* layers,
                                         const fb200_stack_config* stack, int compute, fb200_llama** out) {
  int rc = fb200_bind(dev);
  if (rc) return rc;
  if (!cfg || !layers || !out) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "create_layers: null argument");
  *out = nullptr;
  if (cfg->n_layer <= 0 || cfg->hidden <= 0 || cfg->vocab <= 0 || cfg->max_seq_len <= 0 || cfg->max_batch <= 0 ||
      (compute != FB200_COMPUTE_BF16 && compute != FB200_COMPUTE_F32))
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "create_layers: unsupported configuration");
  for (int i = 0; i < cfg->n_layer; ++i)
    if ((rc = check_mixer(dev, layers, i))) return rc;
  auto* hy = new fb200_hybrid();
  fb200_llama* m = new fb200_llama();
  m->dev = dev;
  m->cfg = *cfg;
  m->cfg.ffn = m->cfg.n_head = m->cfg.n_kv_head = m->cfg.head_dim = 0;
  m->hybrid = hy;
  hy->f32 = compute == FB200_COMPUTE_F32;
  if (stack) hy->stack = *stack;
  hy->mixers.resize(cfg->n_layer);
  for (int i = 0; i < cfg->n_layer; ++i) {
    hy->mixers[i].c = layers[i];
    if (!layers[i].beside) {
      hy->layers.emplace_back();
      hy->layers.back().first = i;
    }
    hy->layers.back().count++;
  }
  const int n = (int)hy->layers.size(), start = hy->stack.loop_start, stop = hy->stack.loop_stop, times = hy->stack.loop_times;
  if (times < 0 || (times && (start < 0 || stop <= start || stop > n)))
    rc = fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "create_layers: %d passes over layers %d .. %d of %d", times, start, stop, n);
  hy->ldx = (size_t)cfg->hidden * (times ? 2 : 1);
  for (int i = 0; i < n && !rc; ++i) {
    if (times && i == start) {
      for (int p = 0; p < times; ++p)
        for (int k = start; k < stop; ++k) hy->runs.push_back({k, p, k == start});
    }
    if (times && i >= start && i < stop) hy->layers[i].passes = times;
    else hy->runs.push_back({i, 0, 0});
  }
  if (!rc) rc = fb200_decoder_session(m);
  for (int i = 0; i < n && !rc; ++i) rc = make_layer(m, i);
  if (rc) {
    fb200_llama_free(m);
    return rc;
  }
  *out = m;
  return FB200_OK;
}
