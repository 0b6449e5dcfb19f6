// Token mixers of the hybrid decoder layers: what a layer's host code hands to the kernels of
// delta_rule.cu, latent_attn.cu, group_attn.cu and linear_attn.cu. Every size and constant is an argument.
#pragma once

#include "common.cuh"

// ---- gated delta rule -------------------------------------------------------------------------------
// Projections [b * s, ldy] hold, per row, q [hk, d] | k [hk, d] | v [h, v] | gate [h, v] | write strength [h] |
// decay [h] at the given columns; q, k and v start at column 0, so that column c of the first
// 2 hk d + h v columns is channel c of the short convolution. The state of a sequence is S, f32
// [h][v][dp] (dp = d padded, see fb200_delta_dp), and the last `taps` inputs of the convolution, f32
// [taps][channels], the input of position p in slot p % taps. Nothing has to be cleared for a new sequence:
// position 0 starts from zero whatever the buffers hold.
struct fb200_delta_args {
  const float* y;
  size_t ldy;
  int off_v, off_g, off_b, off_a;
  const float *conv_w, *a_log, *dt_bias, *out_norm;  // conv_w [taps][channels]
  float eps;
  float *state, *ring;
  int b, s, h, hk, d, v, dp, taps, channels;
  const int* pos_dev;
  void* z;  // [b * s, ldz], h * v columns written
  size_t ldz;
  int z_bf16;
  int commit;  // 0: a dry run of a decode step, the state stays as it is
  // prompt pass scratch: unit q and k [rows][hk][dp], v [rows][h v], (decay, write strength) [rows][h][2],
  // products of four tokens' k and q [b][ceil(s / 4)][hk][16], read-out [rows][h v]
  float *qn, *kn, *vn, *gb, *kq, *o;
};
int fb200_delta_dp(int d);                                         // padded head size, 0 when d is not covered
int fb200_delta_step(fb200_device* dev, const fb200_delta_args& a);    // s == 1: one kernel
int fb200_delta_prompt(fb200_device* dev, const fb200_delta_args& a);  // s > 1

// ---- latent attention --------------------------------------------------------------------------------
// Projections [b * s, ldy]: q [h][d unrotated | r rotated] at column 0, output gate [h] at off_g and, for a layer
// with a cache of its own, the latent's rk + r rows at off_dkv (-1: the cache is another layer's and already
// holds these positions). The cache holds per position the normalised latent (rk) and the rotated key part
// (r), ldc elements apart, bf16 or f32 (cache_f32). w_ukv stacks the key expansion [h d, rk] and the value
// expansion [h v, rk], rkp columns apart. Rotary positions pair dimension i of r with i + r / 2. Query i sees
// the keys j with 0 <= i - j < window (window 0: all of 0 .. i).
struct fb200_latent_args {
  const float* y;
  size_t ldy;
  int off_g, off_dkv;
  const void* w_ukv;
  const float* c_norm;
  float eps;
  void* cache;
  int cache_f32, ldc, cap;
  const float *rope_cos, *rope_sin;  // [cap, r / 2]
  int b, s, h, d, r, v, rk, rkp, window;
  float scale;
  const int* pos_dev;
  int pos;  // the same on the host (prompt passes)
  void* z;
  size_t ldz;
  int z_bf16;
  float *qa, *part;  // [rows][h][rk + r]; [rows][h][nsplit][rk + 2]
  int nsplit;
  __nv_bfloat16* kvx;  // prompt pass with expanded keys and values: [b * keys][h d | h v]
};
bool fb200_latent_covers(int d, int r, int v, int rk);
int fb200_latent_nsplit(const fb200_device* dev, int b, int h, int window, int cap);
int fb200_latent_append(fb200_device* dev, const fb200_latent_args& a);  // the new positions' latents into the cache only
int fb200_latent_rows(fb200_device* dev, const fb200_latent_args& a);    // any s: append, latent-space attention row by row
bool fb200_latent_prefill_covers(int h, int d, int r, int v, int rk, float scale);
int fb200_latent_prefill(fb200_device* dev, const fb200_latent_args& a, const fb200_qmatrix* w_ukv);  // after the append

// ---- grouped softmax attention ---------------------------------------------------------------------------
// Projections [b * s, ldy]: q [h][d] at column 0, k [g][d] at off_k, v [g][v] at off_v, output gate [h] at off_g (-1:
// none). q and k heads are RMS-normalised under q_norm / k_norm (null: not), then rotated on their first r dimensions (i pairs
// with i + r / 2). The cache holds per position k [g][dp] | v [g][vp] (dp, vp: sizes padded to 8, the padding zero), ldc
// elements apart, bf16 or f32. Scores (q . k) scale, through softcap tanh(. / softcap) if softcap > 0; query i sees the keys j
// with 0 <= i - j < window (window 0: all of 0 .. i); sink (null: none) adds exp(sink[head]) to the denominator. The
// output is x sigmoid(gate) x out_scale.
struct fb200_attn_args {
  const float* y;
  size_t ldy;
  int off_k, off_v, off_g;
  const float *q_norm, *k_norm, *sink;
  float eps, scale, softcap, out_scale;
  const float *rope_cos, *rope_sin;  // [cap, r / 2]
  void* cache;
  int cache_f32, ldc, cap;
  int b, s, h, g, d, v, dp, vp, r, window;
  const int* pos_dev;
  int pos;  // the same on the host (prompt passes)
  void* z;
  size_t ldz;
  int z_bf16;
  void* qn;     // prompt passes: prepared queries [rows][h][dp], f32 (rows) or bf16 (tensor cores)
  float* part;  // fb200_attn_part_floats
  int* done;    // [rows * h] arrival counters, zero between launches
};
bool fb200_attn_covers(int d, int v);
size_t fb200_attn_part_floats(const fb200_device* dev, int v);
int fb200_attn_prepare(fb200_device* dev, const fb200_attn_args& a, bool q_bf16);  // queries into qn, keys and values into the cache
int fb200_attn_rows(fb200_device* dev, const fb200_attn_args& a);                  // any s, row by row; s == 1 is one kernel
bool fb200_attn_prefill_covers(int h, int d, int v, float scale);
int fb200_attn_prefill(fb200_device* dev, const fb200_attn_args& a);               // bf16, tensor cores

// ---- linear attention with a fixed decay per head ----------------------------------------------------------
// Projections [b * s, ldy]: q [h][d] at column 0, k [h][d] at off_k, v [h][v] at off_v (all through SiLU), gate [h v] at
// off_g. The state of a sequence is S, f32 [h][v][dp]; position 0 starts from zero whatever the buffer holds. decay
// [h][FB200_LINEAR_CHUNK + 1] holds the powers 0 .. of every head's decay.
constexpr int FB200_LINEAR_CHUNK = 128, FB200_LINEAR_SEGMENTS = 4;
struct fb200_linear_args {
  const float* y;
  size_t ldy;
  int off_k, off_v, off_g;
  const float *decay, *out_norm;
  float eps, out_scale;
  float* state;
  int b, s, h, d, v, dp;
  const int* pos_dev;
  void* z;
  size_t ldz;
  int z_bf16;
  int commit;  // 0: a dry run of a decode step, the state stays as it is
  int bf16;    // prompt operands may be bf16
  float* o;    // read-out [rows][h v]
  int* done;   // [b] arrival counters, zero between launches
  __nv_bfloat16 *q16, *k16, *v16;  // prompt scratch: SiLU'd q, k [rows][h][dp], v [rows][h][vp], vp = v padded to 8
  float* seg;  // prompt scratch: [FB200_LINEAR_SEGMENTS][b][h][v][dp]
};
int fb200_linear_dp(int d);                                              // padded head size, 0 when d is not covered
int fb200_linear_step(fb200_device* dev, const fb200_linear_args& a);    // s == 1: one kernel
int fb200_linear_prompt(fb200_device* dev, const fb200_linear_args& a);  // s > 1
bool fb200_linear_prefill_covers(const fb200_linear_args& a);
int fb200_linear_prefill(fb200_device* dev, const fb200_linear_args& a);  // read-out of a prompt from q16, k16, v16: tensor cores
