// Selective scan: per channel c and state n,  S <- exp(dt A) S + dt x B_n,  y = sum_n S C_n + D x,  out = y silu(z) scale,
// with a step size dt = softplus(W_dt low + bias) and B, C that depend on the position.
#pragma once
#include <cuda_bf16.h>

#include "ugb_internal.h"

// A channel takes np states in memory; the ones behind the model's count have B = C = 0 and stay zero.  In a step they are
// dealt to `lanes` neighbouring lanes with `per_lane` states each.
struct ugb_scan_shape { int lanes, per_lane, np; };
// lanes = 0 when there is no kernel for so many states
ugb_scan_shape ugb_scan_shape_of(int states);
// Factor of the stored A: the bf16 kernels use powers of two.
float ugb_scan_decay_unit(bool f32);

struct ugb_scan_args {
  bool f32;                         // T = f32, else bf16
  ugb_scan_shape shape;
  int channels;                     // padded, a multiple of 8
  const void *u;                    // T [rows][channels]: x
  const float *a;                   // [channels][np]: -exp(A_log) times ugb_scan_decay_unit
  const float *skip, *dt_bias;      // [channels]
  float *state;                     // [b][channels][np], in and out
  void *out;                        // T, rows out_ld apart
  size_t out_ld;
  float scale;
  int xr, rp;                       // columns of low | B | C, of low
};
// A block: t positions of b sequences, rows (b, i).  dt [rows][channels] = W_dt low, xdb [rows][xr], z rows z_ld apart, all T.
int32_t ugb_scan_block(ugb_device *dev, const ugb_scan_args &a, const void *dt, const void *xdb, const void *z, size_t z_ld, int b, int t);
// One position of `rows` sequences: W_dt T [rp][channels]; xdb and z are sums of f32 partials.  early: u, z and the state were
// written by kernels before the predecessor (see row_update_kernel).
struct ugb_scan_partials { const float *p; int n; size_t stride, ld; };
int32_t ugb_scan_step(ugb_device *dev, const ugb_scan_args &a, const void *w_dt, ugb_scan_partials xdb, ugb_scan_partials z, int rows,
                      bool pdl, bool early);
