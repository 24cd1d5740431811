// Attention over a cache of latents: every head's keys and values are linear functions of one cached vector per
// position, so a head's query can be carried into the latent space (q W_uk) and the attention output out of it
// (W_uv o) -- the cache is then one [positions, rank] matrix shared by all heads.
#pragma once
#include <cuda_bf16.h>

#include "ugb_internal.h"

struct ugb_latent_attention_args {
  const void *q;           // [rows][heads][ld]: queries in the latent space (bf16 or f32)
  const void *cache;       // [batch][t_max][ld] of the same type
  void *out;               // [rows][heads][ld] of the same type: softmax-weighted latents times the head's gate
  const float *gate;       // [rows][gate_ld] per-head output factors, null = 1
  int f32;                 // 1: everything f32, 0: bf16 with fp32 scores, softmax and sums
  int rows, t;             // row r = (sequence r / t, position *pos_p + pos_off + r % t)
  const int *pos_p;        // device
  int pos_off;
  int heads, ld, t_max, gate_ld;
  float scale;
  int splits;              // slices of the cached positions per row that run as separate CTAs (bf16 fast path)
  bool pdl;
  bool early;              // with pdl, t == 1: the position and every cache row but the newest were written by kernels that
                           // are complete when this one starts, and may be read before the wait for the preceding one
};

// Row width (elements) the bf16 fast path wants for a latent of `rank` values, or 0 when it has no kernel for it.
int ugb_latent_row_width(int rank);
constexpr int UGB_LATENT_MAX_SPLITS = 8;   // CTAs of a cluster
// Sets the kernels' shared-memory attributes (must not happen inside a stream capture).
int32_t ugb_latent_attention_prepare(ugb_device *dev);
int32_t ugb_latent_attention(ugb_device *dev, const ugb_latent_attention_args &a);
