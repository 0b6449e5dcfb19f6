// Decoder layers made of token mixers (gated delta rule, latent attention) over dense weights.
//
// A layer has one norm whose output feeds everything: h = rms_norm(x), x <- x + (mixer(h) + ffn(h)). So all
// matrices that read h are stacked into one, w_in = [mixer projections | gate | up], and the two that write
// the residual are joined along K, w_out = [mixer output | down]: a layer is
//   product (norm in its prologue for one row; SwiGLU in its epilogue) -> mixer -> product (+ residual).
// One new position of one sequence runs the single-row product with f32 activations; more rows run the tensor-core product
// with bf16 operands, or the f32 product of an F32 model. Steps of one position per sequence are captured
// in a CUDA graph by llama.cu like those of a Llama decoder.
#include <algorithm>
#include <cstring>
#include <memory>

#include "decoder.cuh"
#include "dense.cuh"
#include "mixers.cuh"

void fb200_rope_tables_host(int head_dim, int ctx, float theta, float factor, float low_ff, float high_ff, int original_ctx,
                            const float* freq_weight, std::vector<float>& cs, std::vector<float>& sn);
int fb200_launch_rms_norm_strided(fb200_device* dev, const float* x, size_t x_stride, const float* res, const float* w, float eps,
                                  size_t rows, size_t n, float* y);
int fb200_launch_argmax(fb200_device* dev, const float* logits, size_t rows, size_t n, uint32_t* ids, float* vals);

namespace {

struct MixerLayer {
  fb200_layer_config c{};
  fb200_qmatrix *w_in = nullptr, *w_out = nullptr, *w_ukv = nullptr;
  int n_plain = 0, ko = 0;  // projection rows of the mixer; columns of its output in front of the feed-forward's
  int off_v = 0, off_g = 0, off_b = 0, off_a = 0, off_dkv = -1;
  float* norm = nullptr;
  // delta rule
  int dp = 0, channels = 0;
  float *conv_w = nullptr, *a_log = nullptr, *dt_bias = nullptr, *out_norm = nullptr, *state = nullptr, *ring = nullptr;
  // latent attention
  int rkp = 0, ldc = 0;
  float* c_norm = nullptr;
  void* cache = nullptr;
  float *rope_cos = nullptr, *rope_sin = nullptr;
  bool own_rope = false;
  uint32_t have = 0, need = 0;  // bit per tensor id
};

size_t up_to(size_t n, size_t m) { return (n + m - 1) / m * m; }

}  // namespace

struct fb200_hybrid {
  bool f32 = false;
  std::vector<MixerLayer> layers;
  size_t ldy = 0, ldz = 0;  // widest projection / operand row
  float *proj = nullptr, *zf = nullptr;
  __nv_bfloat16 *hb = nullptr, *zb = nullptr;
  float *qn = nullptr, *kn = nullptr, *vn = nullptr, *gb = nullptr, *kq = nullptr, *o = nullptr;
  float *qa = nullptr, *part = nullptr;
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

int check_layer(fb200_device* dev, const fb200_layer_config* all, int i) {
  const auto& c = all[i];
  if (c.ffn < 0 || c.heads <= 0 || c.dim <= 0 || c.vdim <= 0)
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: ffn %d heads %d dim %d vdim %d", i, c.ffn, c.heads, c.dim, c.vdim);
  if (c.mixer == FB200_MIX_DELTA) {
    if (c.kv_heads <= 0 || c.heads % c.kv_heads || c.conv <= 0 || !fb200_delta_dp(c.dim) || c.vdim > 4096)
      return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: delta rule with %d / %d heads of %d / %d, %d taps", i, c.heads, c.kv_heads,
                        c.dim, c.vdim, c.conv);
    return FB200_OK;
  }
  if (c.mixer != FB200_MIX_LATENT) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d: mixer kind %d", i, c.mixer);
  if (!fb200_latent_covers(c.dim, c.rot_dim, c.vdim, c.kv_rank) || c.window < 0)
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "layer %d: latent attention with dim %d rot_dim %d vdim %d kv_rank %d window %d", i, c.dim,
                      c.rot_dim, c.vdim, c.kv_rank, c.window);
  if (c.kv_from >= 0) {
    if (c.kv_from >= i || all[c.kv_from].mixer != FB200_MIX_LATENT || all[c.kv_from].kv_from >= 0 || all[c.kv_from].kv_rank != c.kv_rank ||
        all[c.kv_from].rot_dim != c.rot_dim || all[c.kv_from].rope_base != c.rope_base)
      return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d: cannot read the latents of layer %d", i, c.kv_from);
  }
  return FB200_OK;
}

int make_layer(fb200_llama* m, int i) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  MixerLayer& L = hy->layers[i];
  const auto& c = L.c;
  const auto& g = m->cfg;
  const size_t E = g.hidden;
  auto need = [&](std::initializer_list<int> ids) { for (int t : ids) L.need |= 1u << t; };
  int rc;
  L.ko = c.heads * c.vdim;
  need({FB200_T_ATTN_NORM, FB200_T_MIX_Q, FB200_T_MIX_GATE, FB200_T_MIX_OUT});
  if (c.ffn) need({FB200_T_FFN_GATE, FB200_T_FFN_UP, FB200_T_FFN_DOWN});
  if (c.mixer == FB200_MIX_DELTA) {
    need({FB200_T_MIX_K, FB200_T_MIX_V, FB200_T_MIX_BETA, FB200_T_MIX_DECAY, FB200_T_MIX_Q_CONV, FB200_T_MIX_K_CONV, FB200_T_MIX_V_CONV,
          FB200_T_MIX_A_LOG, FB200_T_MIX_DT_BIAS, FB200_T_MIX_OUT_NORM});
    L.dp = fb200_delta_dp(c.dim);
    L.off_v = 2 * c.kv_heads * c.dim;
    L.channels = L.off_v + c.heads * c.vdim;
    L.off_g = L.channels;
    L.off_b = L.off_g + c.heads * c.vdim;
    L.off_a = L.off_b + c.heads;
    L.n_plain = L.off_a + c.heads;
    if ((rc = alloc_zero(dev, (void**)&L.conv_w, (size_t)L.channels * c.conv * 4)) || (rc = alloc_zero(dev, (void**)&L.a_log, c.heads * 4)) ||
        (rc = alloc_zero(dev, (void**)&L.dt_bias, c.heads * 4)) || (rc = alloc_zero(dev, (void**)&L.out_norm, c.vdim * 4)) ||
        (rc = alloc_zero(dev, (void**)&L.state, (size_t)g.max_batch * c.heads * c.vdim * L.dp * 4)) ||
        (rc = alloc_zero(dev, (void**)&L.ring, (size_t)g.max_batch * c.conv * L.channels * 4)))
      return rc;
  } else {
    need({FB200_T_MIX_UK, FB200_T_MIX_UV});
    L.rkp = (int)up_to(c.kv_rank, 64);
    L.ldc = (int)up_to(c.kv_rank + c.rot_dim, 8);
    L.off_g = c.heads * (c.dim + c.rot_dim);
    L.n_plain = L.off_g + c.heads;
    if ((rc = make_dense(dev, hy->f32, (uint64_t)c.heads * (c.dim + c.vdim), c.kv_rank, &L.w_ukv))) return rc;
    if (c.kv_from >= 0) {
      L.cache = hy->layers[c.kv_from].cache;
    } else {
      need({FB200_T_MIX_DKV, FB200_T_MIX_DKV_NORM});
      L.off_dkv = L.n_plain;
      L.n_plain += c.kv_rank + c.rot_dim;
      if ((rc = alloc_zero(dev, (void**)&L.c_norm, c.kv_rank * 4)) ||
          (rc = alloc_zero(dev, &L.cache, (size_t)g.max_batch * g.max_seq_len * L.ldc * (hy->f32 ? 4 : 2))))
        return rc;
    }
    for (int j = 0; j < i && !L.rope_cos; ++j) {
      const MixerLayer& P = hy->layers[j];
      if (P.c.mixer == FB200_MIX_LATENT && P.c.rot_dim == c.rot_dim && P.c.rope_base == c.rope_base) { L.rope_cos = P.rope_cos; L.rope_sin = P.rope_sin; }
    }
    if (!L.rope_cos) {
      std::vector<float> cs, sn;
      fb200_rope_tables_host(c.rot_dim, g.max_seq_len, c.rope_base, 0.f, 1.f, 4.f, g.max_seq_len, nullptr, cs, sn);
      L.own_rope = true;
      if ((rc = alloc_zero(dev, (void**)&L.rope_cos, cs.size() * 4)) || (rc = alloc_zero(dev, (void**)&L.rope_sin, sn.size() * 4))) return rc;
      FB_CUDA(dev, cudaMemcpy(L.rope_cos, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice));
      FB_CUDA(dev, cudaMemcpy(L.rope_sin, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice));
    }
  }
  if ((rc = make_dense(dev, hy->f32, (uint64_t)L.n_plain + 2 * c.ffn, E, &L.w_in)) || (rc = make_dense(dev, hy->f32, E, (uint64_t)L.ko + c.ffn, &L.w_out)) ||
      (rc = alloc_zero(dev, (void**)&L.norm, E * 4)))
    return rc;
  hy->ldy = std::max(hy->ldy, up_to(L.n_plain, 8));
  hy->ldz = std::max(hy->ldz, up_to(L.ko + c.ffn, 8));
  return FB200_OK;
}

// A prompt pass long enough for the expansion of keys and values to pay (tensor-core attention over them)
bool expanded(const fb200_hybrid* hy, const fb200_layer_config& c, int seq) {
  return !hy->f32 && seq >= 16 && fb200_latent_prefill_covers(c.heads, c.dim, c.rot_dim, c.vdim, c.kv_rank, c.scale);
}

int run_layer(fb200_llama* m, MixerLayer& L, int batch, int seq, bool commit) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const auto& c = L.c;
  const int rows = batch * seq, E = m->cfg.hidden;
  const bool wide = hy->f32 || rows == 1;  // f32 operand rows
  int rc;
  fb200_dense_job in;
  in.w = L.w_in; in.m = rows; in.kx = E;
  if (rows == 1) {
    in.x = m->x; in.ldx = E; in.norm_w = L.norm; in.eps = m->cfg.rms_eps;
  } else if (hy->f32) {
    if ((rc = fb200_launch_rms_norm_strided(dev, m->x, E, nullptr, L.norm, m->cfg.rms_eps, rows, E, m->xn))) return rc;
    in.x = m->xn; in.ldx = E;
  } else {
    if ((rc = fb200_rows_to_bf16(dev, m->x, E, nullptr, L.norm, m->cfg.rms_eps, rows, E, (int)L.w_in->k, hy->hb))) return rc;
    in.x = hy->hb; in.ldx = L.w_in->k;
  }
  in.n_plain = L.n_plain; in.y = hy->proj; in.ldy = hy->ldy;
  in.gate0 = L.n_plain; in.up0 = L.n_plain + c.ffn; in.ff = c.ffn;
  in.z = wide ? (void*)(hy->zf + L.ko) : (void*)(hy->zb + L.ko); in.ldz = hy->ldz;
  if ((rc = fb200_dense_product(dev, in))) return rc;

  void* z = wide ? (void*)hy->zf : (void*)hy->zb;
  if (c.mixer == FB200_MIX_DELTA) {
    fb200_delta_args a = {};
    a.y = hy->proj; a.ldy = hy->ldy; a.off_v = L.off_v; a.off_g = L.off_g; a.off_b = L.off_b; a.off_a = L.off_a;
    a.conv_w = L.conv_w; a.a_log = L.a_log; a.dt_bias = L.dt_bias; a.out_norm = L.out_norm; a.eps = m->cfg.rms_eps;
    a.state = L.state; a.ring = L.ring; a.b = batch; a.s = seq; a.h = c.heads; a.hk = c.kv_heads; a.d = c.dim; a.v = c.vdim;
    a.dp = L.dp; a.taps = c.conv; a.channels = L.channels; a.pos_dev = m->pos_dev; a.z = z; a.ldz = hy->ldz; a.z_bf16 = !wide; a.commit = commit;
    a.qn = hy->qn; a.kn = hy->kn; a.vn = hy->vn; a.gb = hy->gb; a.kq = hy->kq; a.o = hy->o;
    if ((rc = seq == 1 ? fb200_delta_step(dev, a) : fb200_delta_prompt(dev, a))) return rc;
  } else {
    fb200_latent_args a = {};
    a.y = hy->proj; a.ldy = hy->ldy; a.off_g = L.off_g; a.off_dkv = L.off_dkv; a.w_ukv = L.w_ukv->data; a.c_norm = L.c_norm;
    a.eps = m->cfg.rms_eps; a.cache = L.cache; a.cache_f32 = hy->f32; a.ldc = L.ldc; a.cap = m->cfg.max_seq_len;
    a.rope_cos = L.rope_cos; a.rope_sin = L.rope_sin; a.b = batch; a.s = seq; a.h = c.heads; a.d = c.dim; a.r = c.rot_dim; a.v = c.vdim;
    a.rk = c.kv_rank; a.rkp = L.rkp; a.window = c.window; a.scale = c.scale; a.pos_dev = m->pos_dev; a.pos = m->pos;
    a.z = z; a.ldz = hy->ldz; a.z_bf16 = !wide; a.qa = hy->qa; a.part = hy->part;
    if (expanded(hy, c, seq)) {
      a.kvx = hy->kvx;
      if ((rc = fb200_latent_append(dev, a)) || (rc = fb200_latent_prefill(dev, a, L.w_ukv))) return rc;
    } else {
      a.nsplit = fb200_latent_nsplit(dev, rows, c.heads, c.window, m->cfg.max_seq_len);
      if ((rc = fb200_latent_rows(dev, a))) return rc;
    }
  }

  fb200_dense_job out;
  out.w = L.w_out; out.m = rows; out.x = z; out.ldx = hy->ldz; out.kx = L.ko + c.ffn;
  out.n_plain = E; out.y = m->x; out.ldy = E; out.add = m->x; out.ldadd = E;
  return fb200_dense_product(dev, out);
}

}  // namespace

int fb200_hybrid_ensure_rows(fb200_llama* m, size_t rows) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  const size_t E = m->cfg.hidden;
  size_t qk = 0, hv = 0, heads = 0, kvh = 0, qa = 0, part = 0;
  for (const auto& L : hy->layers) {
    const auto& c = L.c;
    if (c.mixer == FB200_MIX_DELTA) {
      qk = std::max(qk, (size_t)c.kv_heads * L.dp);
      hv = std::max(hv, (size_t)c.heads * c.vdim);
      heads = std::max(heads, (size_t)c.heads);
      kvh = std::max(kvh, (size_t)c.kv_heads);
    } else {
      // rows of the latent-space path: all of them, or fewer where longer passes expand keys and values
      const bool exp = expanded(hy, c, 16);
      const size_t r = exp ? std::min(rows, (size_t)16 * m->cfg.max_batch) : rows;
      qa = std::max(qa, r * c.heads * (size_t)(c.kv_rank + c.rot_dim));
      part = std::max(part, std::max(r * c.heads, (size_t)8 * dev->sm_count) * (size_t)(c.kv_rank + 2));
    }
  }
  struct { void** p; size_t bytes; } bufs[] = {
      {(void**)&m->x, rows * E * 4}, {(void**)&m->xn, rows * E * 4}, {(void**)&hy->proj, rows * hy->ldy * 4}, {(void**)&hy->zf, rows * hy->ldz * 4},
      {(void**)&hy->hb, rows * up_to(E, 64) * 2}, {(void**)&hy->zb, rows * hy->ldz * 2}, {(void**)&hy->qn, rows * qk * 4},
      {(void**)&hy->kn, rows * qk * 4}, {(void**)&hy->vn, rows * hv * 4}, {(void**)&hy->gb, rows * heads * 8}, {(void**)&hy->kq, (rows + 3 * (size_t)m->cfg.max_batch) / 4 * kvh * 64 + 64},
      {(void**)&hy->o, rows * hv * 4}, {(void**)&hy->qa, qa * 4}, {(void**)&hy->part, part * 4}};
  for (auto& b : bufs) {
    if (*b.p) { cudaFree(*b.p); *b.p = nullptr; }
    FB_CUDA(dev, cudaMalloc(b.p, b.bytes ? b.bytes : 16));
    if (dev->poison) FB_CUDA(dev, cudaMemsetAsync(*b.p, 0xFF, b.bytes ? b.bytes : 16, dev->stream));
  }
  return FB200_OK;
}

int fb200_hybrid_finalize(fb200_llama* m) {
  if (!m->output) return fb200_fail(m->dev, FB200_ERR_INVALID_ARGUMENT, "the output head is not set");
  for (size_t i = 0; i < m->hybrid->layers.size(); ++i) {
    const MixerLayer& L = m->hybrid->layers[i];
    if ((L.have & L.need) != L.need)
      return fb200_fail(m->dev, FB200_ERR_INVALID_ARGUMENT, "layer %zu is missing tensors (ids 0x%x)", i, L.need & ~L.have);
  }
  return FB200_OK;
}

int fb200_hybrid_row_logits(fb200_llama* m, size_t row, float* logits_dev) {
  fb200_dense_job j;
  j.w = m->output; j.m = 1; j.x = m->x + row * m->cfg.hidden; j.ldx = m->cfg.hidden; j.kx = m->cfg.hidden;
  j.norm_w = m->output_norm; j.eps = m->cfg.rms_eps; j.n_plain = m->cfg.vocab; j.y = logits_dev; j.ldy = m->cfg.vocab;
  return fb200_dense_product(m->dev, j);
}

int fb200_hybrid_forward(fb200_llama* m, int batch, int seq, bool commit) {
  fb200_device* dev = m->dev;
  fb200_hybrid* hy = m->hybrid;
  int rc;
  size_t kvx = 0;
  for (const auto& L : hy->layers)
    if (L.c.mixer == FB200_MIX_LATENT && expanded(hy, L.c, seq)) {
      const int before = L.c.window && L.c.window - 1 < m->pos ? L.c.window - 1 : m->pos;
      kvx = std::max(kvx, (size_t)batch * (before + seq) * L.c.heads * (L.c.dim + L.c.vdim));
    }
  if (kvx > hy->kvx_elems) {
    FB_CUDA(dev, cudaStreamSynchronize(dev->stream));
    if (hy->kvx) cudaFree(hy->kvx);
    hy->kvx = nullptr;
    hy->kvx_elems = 0;
    FB_CUDA(dev, cudaMalloc(&hy->kvx, kvx * 2));
    hy->kvx_elems = kvx;
  }
  for (auto& L : hy->layers)
    if ((rc = run_layer(m, L, batch, seq, commit))) return rc;
  // final norm and output head on the last position of every sequence
  const int E = m->cfg.hidden;
  if (batch == 1) {
    if ((rc = fb200_hybrid_row_logits(m, (size_t)seq - 1, m->logits))) return rc;
  } else {
    fb200_dense_job j;
    j.w = m->output; j.m = batch; j.kx = E; j.n_plain = m->cfg.vocab; j.y = m->logits; j.ldy = m->cfg.vocab;
    const float* last = m->x + (size_t)(seq - 1) * E;
    if (hy->f32) {
      if ((rc = fb200_launch_rms_norm_strided(dev, last, (size_t)seq * E, nullptr, m->output_norm, m->cfg.rms_eps, batch, E, m->last))) return rc;
      j.x = m->last; j.ldx = E;
    } else {
      if ((rc = fb200_rows_to_bf16(dev, last, (size_t)seq * E, nullptr, m->output_norm, m->cfg.rms_eps, batch, E, (int)m->output->k, hy->hb))) return rc;
      j.x = hy->hb; j.ldx = m->output->k;
    }
    if ((rc = fb200_dense_product(dev, j))) return rc;
  }
  return fb200_launch_argmax(dev, m->logits, batch, m->cfg.vocab, m->next, nullptr);
}

bool fb200_hybrid_recurrent(const fb200_llama* m) {
  if (!m->hybrid) return false;
  for (const auto& L : m->hybrid->layers)
    if (L.c.mixer == FB200_MIX_DELTA) return true;
  return false;
}

void fb200_hybrid_free(fb200_llama* m) {
  fb200_hybrid* hy = m->hybrid;
  if (!hy) return;
  for (auto& L : hy->layers) {
    for (fb200_qmatrix* q : {L.w_in, L.w_out, L.w_ukv})
      if (q) fb200_qmatrix_free(q);
    void* bufs[] = {L.norm, L.conv_w, L.a_log, L.dt_bias, L.out_norm, L.state, L.ring, L.c_norm, L.c.kv_from < 0 ? L.cache : nullptr,
                    L.own_rope ? L.rope_cos : nullptr, L.own_rope ? L.rope_sin : nullptr};
    for (void* b : bufs) if (b) cudaFree(b);
  }
  void* bufs[] = {hy->proj, hy->zf, hy->hb, hy->zb, hy->qn, hy->kn, hy->vn, hy->gb, hy->kq, hy->o, hy->qa, hy->part, hy->kvx};
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
  if (layer < 0 || layer >= (int)hy->layers.size() || which < 0 || which > 31) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d tensor %d", layer, which);
  MixerLayer& L = hy->layers[layer];
  const auto& c = L.c;
  if (!(L.need >> which & 1u)) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "layer %d has no tensor %d", layer, which);
  const bool delta = c.mixer == FB200_MIX_DELTA;
  const uint64_t qk = (uint64_t)c.kv_heads * c.dim, hv = (uint64_t)c.heads * c.vdim;
  fb200_qmatrix* w = L.w_in;
  float* vd = nullptr;
  bool conv = false;
  uint64_t row0 = 0, col0 = 0;
  ek = E;
  switch (which) {
    case FB200_T_ATTN_NORM: en = E; ek = 1; vd = L.norm; break;
    case FB200_T_FFN_GATE: en = c.ffn; row0 = L.n_plain; break;
    case FB200_T_FFN_UP: en = c.ffn; row0 = (uint64_t)L.n_plain + c.ffn; break;
    case FB200_T_FFN_DOWN: en = E; ek = c.ffn; w = L.w_out; col0 = L.ko; break;
    case FB200_T_MIX_OUT: en = E; ek = hv; w = L.w_out; break;
    case FB200_T_MIX_Q: en = delta ? qk : (uint64_t)c.heads * (c.dim + c.rot_dim); break;
    case FB200_T_MIX_K: en = qk; row0 = qk; break;
    case FB200_T_MIX_V: en = hv; row0 = L.off_v; break;
    case FB200_T_MIX_GATE: en = delta ? hv : c.heads; row0 = L.off_g; break;
    case FB200_T_MIX_BETA: en = c.heads; row0 = L.off_b; break;
    case FB200_T_MIX_DECAY: en = c.heads; row0 = L.off_a; break;
    case FB200_T_MIX_DKV: en = (uint64_t)c.kv_rank + c.rot_dim; row0 = L.off_dkv; break;
    case FB200_T_MIX_UK: en = (uint64_t)c.heads * c.dim; ek = c.kv_rank; w = L.w_ukv; break;
    case FB200_T_MIX_UV: en = hv; ek = c.kv_rank; w = L.w_ukv; row0 = (uint64_t)c.heads * c.dim; break;
    case FB200_T_MIX_Q_CONV: en = qk; ek = c.conv; conv = true; break;
    case FB200_T_MIX_K_CONV: en = qk; ek = c.conv; col0 = qk; conv = true; break;
    case FB200_T_MIX_V_CONV: en = hv; ek = c.conv; col0 = 2 * qk; conv = true; break;
    case FB200_T_MIX_A_LOG: en = c.heads; ek = 1; vd = L.a_log; break;
    case FB200_T_MIX_DT_BIAS: en = c.heads; ek = 1; vd = L.dt_bias; break;
    case FB200_T_MIX_OUT_NORM: en = c.vdim; ek = 1; vd = L.out_norm; break;
    case FB200_T_MIX_DKV_NORM: en = c.kv_rank; ek = 1; vd = L.c_norm; break;
    default: return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "tensor id %d", which);
  }
  if ((rc = shape_ok())) return rc;
  if (conv) {  // convolution taps [channels, taps] -> columns col0 .. of [taps][channels]
    std::vector<float> f;
    if ((rc = to_f32(dev, type, src, n * k, f))) return rc;
    std::vector<float> t(f.size());
    for (uint64_t i = 0; i < n; ++i)
      for (uint64_t j = 0; j < k; ++j) t[j * n + i] = f[i * k + j];
    FB_CUDA(dev, cudaMemcpy2D(L.conv_w + col0, (size_t)L.channels * 4, t.data(), n * 4, n * 4, k, cudaMemcpyHostToDevice));
    L.have |= 1u << which;
    return FB200_OK;
  }
  rc = vd ? vec(vd) : put_block(dev, w, row0, col0, type, n, k, src);
  if (!rc) L.have |= 1u << which;
  return rc;
}

extern "C" int fb200_llama_create_layers(fb200_device* dev, const fb200_llama_config* cfg, const fb200_layer_config* layers, int compute,
                                         fb200_llama** out) {
  int rc = fb200_bind(dev);
  if (rc) return rc;
  if (!cfg || !layers || !out) return fb200_fail(dev, FB200_ERR_INVALID_ARGUMENT, "create_layers: null argument");
  *out = nullptr;
  if (cfg->n_layer <= 0 || cfg->hidden <= 0 || cfg->vocab <= 0 || cfg->max_seq_len <= 0 || cfg->max_batch <= 0 ||
      (compute != FB200_COMPUTE_BF16 && compute != FB200_COMPUTE_F32))
    return fb200_fail(dev, FB200_ERR_INVALID_SHAPE, "create_layers: unsupported configuration");
  for (int i = 0; i < cfg->n_layer; ++i)
    if ((rc = check_layer(dev, layers, i))) return rc;
  fb200_llama* m = new fb200_llama();
  m->dev = dev;
  m->cfg = *cfg;
  m->cfg.ffn = m->cfg.n_head = m->cfg.n_kv_head = m->cfg.head_dim = 0;
  m->hybrid = new fb200_hybrid();
  m->hybrid->f32 = compute == FB200_COMPUTE_F32;
  m->hybrid->layers.resize(cfg->n_layer);
  rc = fb200_decoder_session(m);
  for (int i = 0; i < cfg->n_layer && !rc; ++i) {
    m->hybrid->layers[i].c = layers[i];
    rc = make_layer(m, i);
  }
  if (rc) {
    fb200_llama_free(m);
    return rc;
  }
  *out = m;
  return FB200_OK;
}
