// Arguments of attention over a paged cache of latents (latent_decode.cu) and of the per-head matrix products around it
// (head_product.cu), mirrored by ctypes structures in ops/latent_attention.py.
//
// One layer's cache is [num_blocks, 64, R]: a token leaves one row c = rms_norm(gain * x[c_off : c_off + R]) * c_norm, which
// all heads share.  With absorbed queries qa[t, h] (R wide) the score of key j is qa . c_j * scale * gain and the result is
// the weighted sum of the c_j.
#pragma once

namespace sb {

struct LatentParams {
  const void* x;            // projected rows [T, row_stride], latents before their norm at c_off
  long long row_stride;
  int c_off, T;
  const int* seq_ids;       // [T] cache slot of every row (-1: none)
  const int* positions;     // [T]
  const int* block_table;   // [slots, max_blocks]
  void* cache;
  long long num_blocks;
  int max_blocks, H, R;
  float scale, eps;
  int pad_;
  const void* c_norm;       // [R]
  const void* gain;         // one number, or null
  const void* qa;           // [T, H, R]
  void* out;                // [T, H, R]
};
static_assert(sizeof(LatentParams) == 120, "LatentParams is mirrored from Python");

// out[t, h, :] = a[t, h, :] * B_h for every head: B_h [b_rows, b_cols] row-major, heads stacked.
// b_mn 1: contraction over the rows of B_h (N = b_cols); 0: over its columns (N = b_rows).
struct HeadProduct {
  const void* a;
  long long a_head, a_row;  // pitches of heads and rows, in elements
  const void* b;
  int b_rows, b_cols, b_mn, T, H, pad_;
  void* c;                  // [T, c_row], head h at column h * N
  long long c_row;
  const void* gate;         // columns like c's: the result is multiplied by sigmoid(gain * gate); null: none
  long long gate_row;
  const void* gain;         // one number, or null
};
static_assert(sizeof(HeadProduct) == 96, "HeadProduct is mirrored from Python");

}  // namespace sb
