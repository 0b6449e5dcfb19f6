// Token mixers of the hybrid decoder layers: what a layer's host code hands to the kernels of
// delta_rule.cu and latent_attn.cu. Every size and constant is an argument.
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
