// Gated outer-product recurrences (linear attention with a matrix state), for prefill and for decode.
//
//   S_t = diag(a_t) S_(t-1) + w_t k_t v_t^T          o_t = S_t^T q_t
//
// per sequence and head, with the state in 32-bit floats.  Two gate forms share the kernels:
//   kGateChannel  a_t = sigmoid(W2 (low-rank row) + b)^(1 / tau) per key channel, w_t = 1
//   kGateHead     scalar gates of a stabilised matrix memory: with i = cap tanh(i_pre / cap) and
//                 f = logsigmoid(cap tanh(f_pre / cap)), m_t = max(f + m_(t-1), i), a_t = exp(f + m_(t-1) - m_t),
//                 w_t = exp(i - m_t); a normaliser n with the same recurrence is the extra value column v = 1, and
//                 o_t is divided by max(|n . q|, exp(-m_t)) + 1e-6
// followed by an RMS norm over the head's values, a norm weight (shared by the heads or per head), an output gate
// (SiLU or sigmoid of a projected row) and a scale.
//
// State layout: S [slots, heads, dv (+1 for the normaliser), dk] fp32 (value-major: a row holds one value column's key
// channels), m [slots, heads].  A portion whose first position is 0 starts from the zero state and does not read its
// slot, so a slot that is used again needs no clearing.
//
// Kernels:
//   recurrence_step_kernel   any sizes and formats, one CTA per (sequence, head), token by token: decode (one token: the
//                            state is streamed once) and the general prefill path (state in shared memory if it fits)
//   gate_scan_kernel         prefill, kGateHead: m_t of a whole portion by a block-wide scan of max-plus affine maps
//   chunk_prepare_kernel     prefill: everything of a 16-token chunk that does not depend on the state, in parallel over
//                            chunks and heads: q and k scaled by their decays to the chunk's start / end, the 16 x 16
//                            matrix of decayed scores, the decay of the whole chunk
//   chunk_scan_kernel        prefill: walks the chunks of a segment of one (sequence, head) with the state in registers
//                            as tensor-core fragments; tiles arrive through a ring of asynchronous copies.  Long prompts
//                            are cut into segments that run in parallel: a first pass makes each segment's state from
//                            zero, segment_states_kernel chains them, a second pass makes the outputs
// All decays are formed as exp2 of differences <= 0, so any gate value is safe.  Tensor-core operands that stand for
// 32-bit quantities (decayed q and k, decayed scores, the state) are split into two bf16 terms (16 mantissa bits), v is
// bf16 as projected; accumulation is fp32.
#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"

namespace sb {

enum { kGateChannel = 0, kGateHead = 1 };
constexpr int kChunk = 16;
constexpr float kLog2e = 1.4426950408889634f;

struct RecParams {
  const void* x;               // projected rows [T, row_stride]
  long long row_stride;
  int q_off, k_off, v_off, g_off;
  int e_off, f_off;            // kGateChannel: low-rank row at e_off; kGateHead: i_pre at e_off, f_pre at f_off (per head)
  int kind, rank, norm_per_head, gate_act;   // gate_act: 0 SiLU, 1 sigmoid
  const void* w2;              // [H * dk, rank]
  const void* b_e;             // kGateChannel: [H * dk]; kGateHead: input-gate bias [H]
  const void* b_f;             // kGateHead: forget-gate bias [H]
  const void* norm_w;
  float inv_tau, cap, q_scale, eps, out_scale;
  float* S;
  float* m;
  void* out;                   // [T, out_stride], this branch at column out_off
  long long out_stride;
  int out_off, H, dk, dv;
};

__device__ __forceinline__ float log_sigmoid(float x) {
  return x >= 0.f ? -log1pf(expf(-x)) : x - log1pf(expf(x));
}
__device__ __forceinline__ float gate_value(float g, int act) {
  const float s = 1.f / (1.f + expf(-g));
  return act == 0 ? g * s : s;
}
template <typename T>
__device__ __forceinline__ void head_gates(const RecParams& p, const T* xr, int h, float& i, float& f) {
  const float zi = to_float(xr[p.e_off + h]) + to_float(reinterpret_cast<const T*>(p.b_e)[h]);
  const float zf = to_float(xr[p.f_off + h]) + to_float(reinterpret_cast<const T*>(p.b_f)[h]);
  i = p.cap * tanhf(zi / p.cap);
  f = log_sigmoid(p.cap * tanhf(zf / p.cap));
}

constexpr int kStepThreads = 256;

// V: key channels per access (4 when dk is a multiple of 4)
template <typename T, int V>
__global__ void __launch_bounds__(kStepThreads)
recurrence_step_kernel(RecParams p, const int* __restrict__ row0, const int* __restrict__ nrow,
                       const int* __restrict__ slots, const int* __restrict__ pos0, int smem_state) {
  extern __shared__ __align__(16) float sm[];
  const int dkp = (p.dk + 3) & ~3;
  float* sq = sm;
  float* sk = sq + dkp;
  float* sd = sk + dkp;
  float* so = sd + dkp;
  float* red = so + ((p.dv + 1 + 3) & ~3);
  float* sst = red + 8;
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int rows = p.dv + norm;
  const int r0 = row0 ? row0[s] : s, n = nrow ? nrow[s] : 1, slot = slots[s];
  T* out = reinterpret_cast<T*>(p.out) + p.out_off + (size_t)h * p.dv;
  if (slot < 0) {
    for (int t = 0; t < n; ++t)
      for (int i = tid; i < p.dv; i += kStepThreads) out[(size_t)(r0 + t) * p.out_stride + i] = from_float<T>(0.f);
    return;
  }
  if (n <= 0) return;
  const bool fresh = pos0[s] == 0;
  float* gs = p.S + ((size_t)slot * p.H + h) * rows * p.dk;
  float m = 0.f;
  if (norm && !fresh) m = p.m[(size_t)slot * p.H + h];
  float* st = gs;
  if (smem_state) {
    st = sst;
    for (int i = tid; i < rows * p.dk; i += kStepThreads) sst[i] = fresh ? 0.f : gs[i];
  }
  const int warp = tid >> 5, lane = tid & 31, grp = lane >> 3, l8 = lane & 7;
  for (int t = 0; t < n; ++t) {
    const T* xr = reinterpret_cast<const T*>(p.x) + (size_t)(r0 + t) * p.row_stride;
    float keep = 1.f, put = 1.f;
    if (norm) {
      float i, f;
      head_gates<T>(p, xr, h, i, f);
      const float mn = fmaxf(f + m, i);
      keep = expf(f + m - mn);
      put = expf(i - mn);
      m = mn;
    }
    for (int d = tid; d < p.dk; d += kStepThreads) {
      sq[d] = to_float(xr[p.q_off + h * p.dk + d]) * p.q_scale;
      sk[d] = to_float(xr[p.k_off + h * p.dk + d]) * put;
      float a = keep;
      if (!norm) {
        const T* w = reinterpret_cast<const T*>(p.w2) + (size_t)(h * p.dk + d) * p.rank;
        float z = to_float(reinterpret_cast<const T*>(p.b_e)[h * p.dk + d]);
        for (int r = 0; r < p.rank; ++r) z = fmaf(to_float(w[r]), to_float(xr[p.e_off + r]), z);
        a = expf(log_sigmoid(z) * p.inv_tau);
      }
      sd[d] = a;
    }
    __syncthreads();
    const bool zero = fresh && t == 0 && !smem_state;
    for (int rb = warp * 4; rb < rows; rb += kStepThreads / 8) {
      const int r = rb + grp;
      float dot = 0.f;
      if (r < rows) {
        const float v = r < p.dv ? to_float(xr[p.v_off + h * p.dv + r]) : 1.f;
        float* sr = st + (size_t)r * p.dk;
#pragma unroll 4
        for (int d = l8 * V; d < p.dk; d += 8 * V) {
          float x[V];
          if (zero) {
#pragma unroll
            for (int j = 0; j < V; ++j) x[j] = 0.f;
          } else {
            load_vec<float, V>(sr + d, x);
          }
#pragma unroll
          for (int j = 0; j < V; ++j) {
            x[j] = fmaf(x[j], sd[d + j], sk[d + j] * v);
            dot = fmaf(x[j], sq[d + j], dot);
          }
          store_vec<float, V>(sr + d, x);
        }
      }
      dot += __shfl_xor_sync(0xffffffffu, dot, 4);
      dot += __shfl_xor_sync(0xffffffffu, dot, 2);
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      if (l8 == 0 && r < rows) so[r] = dot;
    }
    __syncthreads();
    float inv = 1.f;
    if (norm) inv = 1.f / (fmaxf(fabsf(so[p.dv]), expf(-m)) + 1e-6f);
    float ss = 0.f;
    for (int i = tid; i < p.dv; i += kStepThreads) {
      const float o = so[i] * inv;
      ss += o * o;
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) tot += red[i];
    const float rstd = 1.f / sqrtf(tot / (float)p.dv + p.eps);
    for (int i = tid; i < p.dv; i += kStepThreads) {
      const float w = to_float(reinterpret_cast<const T*>(p.norm_w)[p.norm_per_head ? h * p.dv + i : i]);
      const float g = gate_value(to_float(xr[p.g_off + h * p.dv + i]), p.gate_act);
      out[(size_t)(r0 + t) * p.out_stride + i] = from_float<T>(so[i] * inv * rstd * w * g * p.out_scale);
    }
  }
  if (smem_state)
    for (int i = tid; i < rows * p.dk; i += kStepThreads) gs[i] = sst[i];
  if (norm && tid == 0) p.m[(size_t)slot * p.H + h] = m;
}

// ---------------------------------------------------------------------------------------
// prefill: m_t by a scan.  Token t is the map m -> max(m + f_t, i_t); maps compose as
// (F1, M1) then (F2, M2) = (F1 + F2, max(M1 + F2, M2)).
// gates[T, H] receives (log a_t, log w_t, exp(-m_t), unused).
// ---------------------------------------------------------------------------------------
constexpr int kGsThreads = 256, kGsPer = 4;

__global__ void __launch_bounds__(kGsThreads)
gate_scan_kernel(RecParams p, const int* __restrict__ row0, const int* __restrict__ nrow, const int* __restrict__ slots,
                 const int* __restrict__ pos0, float4* __restrict__ gates) {
  __shared__ float wf[kGsThreads / 32], wm[kGsThreads / 32], last;
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int r0 = row0[s], n = nrow[s], slot = slots[s];
  if (slot < 0) return;
  float carry = pos0[s] == 0 ? 0.f : p.m[(size_t)slot * p.H + h];
  for (int base = 0; base < n; base += kGsThreads * kGsPer) {
    float f[kGsPer], in[kGsPer];
    float F = 0.f, M = -INFINITY;
#pragma unroll
    for (int j = 0; j < kGsPer; ++j) {
      const int t = base + tid * kGsPer + j;
      f[j] = 0.f;
      in[j] = -INFINITY;
      if (t < n)
        head_gates<__nv_bfloat16>(p, reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)(r0 + t) * p.row_stride, h,
                                  in[j], f[j]);
      M = fmaxf(M + f[j], in[j]);
      F += f[j];
    }
    // inclusive scan over the lanes, then over the warps
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmaxf(Mp + F, M);
        F += Fp;
      }
    }
    __syncthreads();
    if (lane == 31) {
      wf[warp] = F;
      wm[warp] = M;
    }
    __syncthreads();
    float Fe = __shfl_up_sync(0xffffffffu, F, 1), Me = __shfl_up_sync(0xffffffffu, M, 1);
    if (lane == 0) {
      Fe = 0.f;
      Me = -INFINITY;
    }
    float m = carry;
    for (int w = 0; w < warp; ++w) m = fmaxf(m + wf[w], wm[w]);
    m = fmaxf(m + Fe, Me);
#pragma unroll
    for (int j = 0; j < kGsPer; ++j) {
      const int t = base + tid * kGsPer + j;
      const float mn = fmaxf(f[j] + m, in[j]);
      if (t < n) gates[(size_t)(r0 + t) * p.H + h] = make_float4(f[j] + m - mn, in[j] - mn, expf(-mn), 0.f);
      m = mn;
    }
    if (tid == kGsThreads - 1) last = m;
    __syncthreads();
    carry = last;
  }
  if (tid == 0 && n > 0) p.m[(size_t)slot * p.H + h] = carry;
}

// ---------------------------------------------------------------------------------------
// chunk tiles
// ---------------------------------------------------------------------------------------
__host__ __device__ inline int tile_row(int dkp) { return dkp + 8; }        // bf16 elements per row of a q / k tile
constexpr int kARow = 24;                                                    // and of the score matrix
__host__ __device__ inline int tile_bytes(int dkp) {
  return 4 * kChunk * tile_row(dkp) * 2 + 2 * kChunk * kARow * 2 + dkp * 4 + kChunk * 4;
}

// x and y as two bf16 terms each: x = hi + lo to 16 mantissa bits
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16x2(x - f.x, y - f.y);
}

constexpr int kPrepThreads = 128;

// NK: key channels in steps of 16 (padded); SCALAR: one decay per head and token (kGateHead) or one per channel
template <int NK, bool SCALAR>
__global__ void __launch_bounds__(kPrepThreads)
chunk_prepare_kernel(RecParams p, const int* __restrict__ chunk_row, const int* __restrict__ chunk_len,
                     const float4* __restrict__ gates, uint8_t* __restrict__ tiles, int vec) {
  constexpr int dkp = NK * 16, ld = dkp + 1, rs = dkp + 8;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                       // [16][ld]
  float* sk = sq + kChunk * ld;
  float* sc = sk + kChunk * ld;         // log2 of the decay from the chunk's start through token t
  float* sA = sc + kChunk * ld;         // [16][16]
  float* sg = sA + kChunk * kChunk;     // [16][2] log2 decay and write weight of the tokens (SCALAR)
  float* se = sg + kChunk * 2;          // low-rank rows [16][rank]
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row = chunk_row[c], len = chunk_len[c];
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)row * p.row_stride;
  uint8_t* tile = tiles + ((size_t)c * p.H + h) * tile_bytes(dkp);
  __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(tile);
  __nv_bfloat16* ql = qh + kChunk * rs;
  __nv_bfloat16* kh = ql + kChunk * rs;
  __nv_bfloat16* kl = kh + kChunk * rs;
  __nv_bfloat16* Ah = kl + kChunk * rs;
  __nv_bfloat16* Al = Ah + kChunk * kARow;
  float* D = reinterpret_cast<float*>(Al + kChunk * kARow);
  float* floor_ = D + dkp;

  for (int i = tid; i < kChunk * kChunk; i += kPrepThreads) sA[i] = 0.f;
  if (vec) {
    for (int i = tid; i < kChunk * (dkp / 8); i += kPrepThreads) {
      const int t = i / (dkp / 8), d = i % (dkp / 8) * 8;
      float q[8] = {}, k[8] = {};
      if (t < len && d < p.dk) {
        const __nv_bfloat16* xr = x + (size_t)t * p.row_stride + h * p.dk + d;
        load_vec<__nv_bfloat16, 8>(xr + p.q_off, q);
        load_vec<__nv_bfloat16, 8>(xr + p.k_off, k);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        sq[t * ld + d + j] = q[j] * p.q_scale;
        sk[t * ld + d + j] = k[j];
      }
    }
  } else {
    for (int i = tid; i < kChunk * dkp; i += kPrepThreads) {
      const int t = i / dkp, d = i % dkp;
      float q = 0.f, k = 0.f;
      if (t < len && d < p.dk) {
        const __nv_bfloat16* xr = x + (size_t)t * p.row_stride + h * p.dk + d;
        q = to_float(xr[p.q_off]) * p.q_scale;
        k = to_float(xr[p.k_off]);
      }
      sq[t * ld + d] = q;
      sk[t * ld + d] = k;
    }
  }
  if constexpr (SCALAR) {
    if (tid < kChunk) {
      float4 g = make_float4(0.f, 0.f, 1.f, 0.f);
      if (tid < len) g = gates[(size_t)(row + tid) * p.H + h];
      sg[2 * tid] = g.x * kLog2e;
      sg[2 * tid + 1] = expf(g.y);
      floor_[tid] = g.z;
    }
  } else {
    if (tid < kChunk) floor_[tid] = 1.f;
    for (int i = tid; i < kChunk * p.rank; i += kPrepThreads) {
      const int t = i / p.rank;
      se[i] = t < len ? to_float(x[(size_t)t * p.row_stride + p.e_off + i - t * p.rank]) : 0.f;
    }
  }
  __syncthreads();
  if constexpr (!SCALAR) {
    // log decays of (channel, group of 8 tokens) items, then running sums per channel
    for (int i = tid; i < dkp * 2; i += kPrepThreads) {
      const int d = i % dkp, t0 = i / dkp * 8;
      const bool ok = d < p.dk;
      const float b = ok ? to_float(reinterpret_cast<const __nv_bfloat16*>(p.b_e)[h * p.dk + d]) : 0.f;
      float z[8];
#pragma unroll
      for (int t = 0; t < 8; ++t) z[t] = b;
      const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w2) + (size_t)(h * p.dk + (ok ? d : 0)) * p.rank;
#pragma unroll 4
      for (int r = 0; r < p.rank; ++r) {
        const float wr = to_float(w[r]);
#pragma unroll
        for (int t = 0; t < 8; ++t) z[t] = fmaf(wr, se[(t0 + t) * p.rank + r], z[t]);
      }
#pragma unroll
      for (int t = 0; t < 8; ++t)
        sc[(t0 + t) * ld + d] = (t0 + t < len && ok) ? log_sigmoid(z[t]) * p.inv_tau * kLog2e : 0.f;
    }
    __syncthreads();
  }
  for (int d = tid; d < dkp; d += kPrepThreads) {
    float acc = 0.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      if constexpr (SCALAR) sk[t * ld + d] *= sg[2 * t + 1];
      acc += SCALAR ? sg[2 * t] : sc[t * ld + d];
      sc[t * ld + d] = acc;
    }
    D[d] = exp2f(acc);
  }
  __syncthreads();
  // decayed q (to the chunk's start) and k (to its end)
  for (int i = tid; i < kChunk * (dkp / 2); i += kPrepThreads) {
    const int t = i / (dkp / 2), d = i % (dkp / 2) * 2;
    const float c0 = sc[t * ld + d], c1 = sc[t * ld + d + 1];
    const float e0 = sc[(kChunk - 1) * ld + d], e1 = sc[(kChunk - 1) * ld + d + 1];
    uint32_t hi, lo;
    split_pair(sq[t * ld + d] * exp2f(c0), sq[t * ld + d + 1] * exp2f(c1), hi, lo);
    *reinterpret_cast<uint32_t*>(qh + t * rs + d) = hi;
    *reinterpret_cast<uint32_t*>(ql + t * rs + d) = lo;
    split_pair(sk[t * ld + d] * exp2f(e0 - c0), sk[t * ld + d + 1] * exp2f(e1 - c1), hi, lo);
    *reinterpret_cast<uint32_t*>(kh + t * rs + d) = hi;
    *reinterpret_cast<uint32_t*>(kl + t * rs + d) = lo;
  }
  // scores of the chunk with itself: 4 x 4 blocks of (t, s), lanes over the key channels.  Below the diagonal the decay
  // is split at the token before the block's rows, so both factors are at most one.
  for (int blk = warp; blk < 10; blk += kPrepThreads / 32) {
    const int bi = blk < 1 ? 0 : (blk < 3 ? 1 : (blk < 6 ? 2 : 3));
    const int bj = blk - bi * (bi + 1) / 2;
    float a[16] = {};
#pragma unroll
    for (int d0 = 0; d0 < dkp; d0 += 32) {
      const int d = d0 + lane;
      if (dkp % 32 && d >= dkp) break;
      float q[4], k[4], ct[4], cs[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        q[i] = sq[(bi * 4 + i) * ld + d];
        k[i] = sk[(bj * 4 + i) * ld + d];
        if constexpr (!SCALAR) {
          ct[i] = sc[(bi * 4 + i) * ld + d];
          cs[i] = sc[(bj * 4 + i) * ld + d];
        }
      }
      if (SCALAR || bi > bj) {
        if constexpr (!SCALAR) {
          const float anchor = sc[(bi * 4 - 1) * ld + d];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            q[i] *= exp2f(ct[i] - anchor);
            k[i] *= exp2f(anchor - cs[i]);
          }
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) a[i] = fmaf(q[i / 4], k[i % 4], a[i]);
      } else {
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (i % 4 <= i / 4) a[i] = fmaf(q[i / 4] * k[i % 4], i / 4 == i % 4 ? 1.f : exp2f(ct[i / 4] - cs[i % 4]), a[i]);
      }
    }
    // sum over the lanes while halving the values each lane keeps: lane l ends with value l / 2 (both of a pair)
#pragma unroll
    for (int w = 16, n = 8; n >= 1; w >>= 1, n >>= 1) {
      const bool up = lane & w;
#pragma unroll
      for (int i = 0; i < n; ++i) {
        const float keep = up ? a[i + n] : a[i], give = up ? a[i] : a[i + n];
        a[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
      }
    }
    const float v = a[0] + __shfl_xor_sync(0xffffffffu, a[0], 1);
    const int t = bi * 4 + (lane >> 3), s = bj * 4 + ((lane >> 1) & 3);
    if (!(lane & 1) && s <= t) sA[t * kChunk + s] = SCALAR ? v * exp2f(sc[t * ld] - sc[s * ld]) : v;
  }
  __syncthreads();
  {
    const int t = tid >> 3, s = (tid & 7) * 2;
    uint32_t hi, lo;
    split_pair(sA[t * kChunk + s], sA[t * kChunk + s + 1], hi, lo);
    *reinterpret_cast<uint32_t*>(Ah + t * kARow + s) = hi;
    *reinterpret_cast<uint32_t*>(Al + t * kARow + s) = lo;
  }
}

// ---------------------------------------------------------------------------------------
// chunk scan.  A portion is cut into segments of consecutive chunks.  With more than one segment:
//   pass 0  every segment but the last: its state from a zero start, and its whole decay, to the workspace
//   segment_states_kernel  the start state of every segment, element by element along the segments
//   pass 1  every segment from its start state: outputs; the last one leaves the state in the slot
// ---------------------------------------------------------------------------------------
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int kScanStages = 3;
constexpr int kScanMaxWarps = 12;

struct ScanSmem {
  int tile, v_row, v_off, g_off, stage, obuf_off, obuf_row, total;
  __host__ __device__ ScanSmem(int dkp, int dvp, int dv) {
    tile = tile_bytes(dkp);
    v_row = dvp + 8;
    v_off = tile;
    g_off = v_off + kChunk * v_row * 2;
    stage = (g_off + kChunk * dv * 2 + 127) / 128 * 128;
    obuf_off = kScanStages * stage;
    obuf_row = dvp + 4;
    total = obuf_off + kChunk * obuf_row * 4;
  }
};

struct Segments {
  const int* seq;       // [n] sequence of the segment
  const int* chunk0;    // [n] its first chunk
  const int* row;       // [n] its first row
  const int* tokens;    // [n] its tokens
  const int* flags;     // [n] bit 0: first of its sequence, bit 1: last
  const int* seq_seg0;  // [n_seq + 1]
  float* S;             // [n, H, rows, dk] local states, then start states
  float* decay;         // [n, H, dkp]
};

// warp w of the CTA owns value columns 16 w .. 16 w + 15 (rows of the fragment), all key channels (NK steps of 16)
template <int NK, bool OUT>
__global__ void __launch_bounds__(32 * kScanMaxWarps)
chunk_scan_kernel(RecParams p, Segments sg, const int* __restrict__ slots, const int* __restrict__ pos0,
                  const uint8_t* __restrict__ tiles) {
  constexpr int dkp = NK * 16, rs = dkp + 8;
  constexpr int kStateBytes = 2 * kChunk * rs * 2;           // the decayed keys start here in a tile
  constexpr int kDOff = 4 * kChunk * rs * 2 + 2 * kChunk * kARow * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int dvp = (p.dv + norm + 15) / 16 * 16;
  const ScanSmem L(dkp, dvp, p.dv);
  float* ob = reinterpret_cast<float*>(smem + L.obuf_off);
  const int h = blockIdx.x, g_id = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_warps = blockDim.x >> 5;
  const int s = sg.seq[g_id], slot = slots[s], flags = sg.flags[g_id];
  if (slot < 0 || (!OUT && (flags & 2))) return;
  const int tokens = sg.tokens[g_id], n = (tokens + kChunk - 1) / kChunk, row0 = sg.row[g_id];
  const uint8_t* my_tiles = tiles + ((size_t)sg.chunk0[g_id] * p.H + h) * L.tile;
  const size_t tile_step = (size_t)p.H * L.tile;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)row0 * p.row_stride + h * p.dv;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)row0 * p.out_stride + p.out_off + (size_t)h * p.dv;

  // columns of the value tiles that no copy writes: zeros, and ones for the normaliser
  for (int st = 0; st < kScanStages; ++st) {
    __nv_bfloat16* v = reinterpret_cast<__nv_bfloat16*>(smem + st * L.stage + L.v_off);
    const int extra = L.v_row - p.dv;
    for (int i = tid; i < kChunk * extra; i += blockDim.x)
      v[i / extra * L.v_row + p.dv + i % extra] = __float2bfloat16(norm && i % extra == 0 ? 1.f : 0.f);
  }
  const int vv = p.dv / 8;
  const int vshift = 31 - __clz(vv), vpow = (1 << vshift) == vv;      // rows of a power of two vectors: no division
  auto issue = [&](int c) {      // copies of chunk c into its stage (an empty group past the end)
    if (c < n) {
      uint8_t* st = smem + (c % kScanStages) * L.stage;
      const uint8_t* src = my_tiles + (size_t)c * tile_step;
      for (int i = tid * 16 + (OUT ? 0 : kStateBytes); i < L.tile; i += blockDim.x * 16) copy16(st + i, src + i);
      const int len = min(kChunk, tokens - c * kChunk);
      for (int i = tid; i < kChunk * vv; i += blockDim.x) {
        const int t = vpow ? i >> vshift : i / vv, e = (i - t * vv) * 8;
        uint8_t* dst = st + L.v_off + (t * L.v_row + e) * 2;
        if (t < len) {
          const __nv_bfloat16* xr = x + (size_t)(c * kChunk + t) * p.row_stride + e;
          copy16(dst, xr + p.v_off);
          if (OUT) copy16(st + L.g_off + (t * p.dv + e) * 2, xr + p.g_off);
        } else {
          *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
      }
    }
    copy_commit();
  };
#pragma unroll
  for (int i = 0; i < kScanStages - 1; ++i) issue(i);

  // state fragments: acc[j] holds key channels 8 j + 2 (lane % 4) + {0, 1} of value columns r and r + 8
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  const int r = warp * 16 + g;
  const int rows = p.dv + norm;
  float* slot_S = p.S + ((size_t)slot * p.H + h) * rows * p.dk;
  float* seg_S = sg.S + ((size_t)g_id * p.H + h) * rows * p.dk;
  const bool single = (flags & 3) == 3;
  const float* from = single ? slot_S : seg_S;
  const bool zero = !OUT || (single && pos0[s] == 0);
  float acc[2 * NK][4];
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = r + (i >> 1) * 8, d = 8 * j + q2 + (i & 1);
      acc[j][i] = (!zero && rr < rows && d < p.dk) ? from[(size_t)rr * p.dk + d] : 0.f;
    }
  float2 nw[kScanMaxWarps * 16 / 64];      // this lane's norm weights
  if constexpr (OUT) {
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.norm_w) + (p.norm_per_head ? h * p.dv : 0);
#pragma unroll
    for (int k = 0; k < kScanMaxWarps * 16 / 64; ++k) {
      const int i = lane * 2 + k * 64;
      nw[k] = i < p.dv ? __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(w + i)) : make_float2(0.f, 0.f);
    }
  }
  float whole[(dkp + 31) / 32];            // pass 0, warp 0: product of the chunks' decays
#pragma unroll
  for (int k = 0; k < (dkp + 31) / 32; ++k) whole[k] = 1.f;

  // lane's row / column offsets inside a 16 x 16 tile for the ldmatrix arrangements
  const int nrm_row = (lane & 7) + ((lane >> 4) << 3), nrm_col = ((lane >> 3) & 1) * 8;   // pairs along n, then k
  const int trn_row = (lane & 7) + (((lane >> 3) & 1) << 3), trn_col = (lane >> 4) * 8;   // k rows, then n columns
  for (int c = 0; c < n; ++c) {
    copy_wait<kScanStages - 2>();
    __syncthreads();            // chunk c has landed; every warp is through with chunk c - 1 and its stage
    issue(c + kScanStages - 1);
    const uint8_t* st = smem + (c % kScanStages) * L.stage;
    const uint32_t aq = smem_u32(st), al = aq + kChunk * rs * 2, akh = al + kChunk * rs * 2, akl = akh + kChunk * rs * 2;
    const float* D = reinterpret_cast<const float*>(st + kDOff);
    uint32_t va[4];             // v^T: value columns x tokens (rows and columns swap roles with the plain arrangement)
    ldsm_x4_t(va, smem_u32(st + L.v_off) + (uint32_t)(nrm_row * L.v_row + warp * 16 + nrm_col) * 2);
    if constexpr (OUT) {
      const uint32_t aA = akl + kChunk * rs * 2, aAl = aA + kChunk * kARow * 2;
      float o0[2][4] = {}, o1[2][4] = {}, o2[2][4] = {};
#pragma unroll
      for (int kk = 0; kk < NK; ++kk) {
        uint32_t hi[4], lo[4], bh[4], bl[4];
        const uint32_t off = (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2;
        ldsm_x4(bh, aq + off);
        ldsm_x4(bl, al + off);
        split_pair(acc[2 * kk][0], acc[2 * kk][1], hi[0], lo[0]);
        split_pair(acc[2 * kk][2], acc[2 * kk][3], hi[1], lo[1]);
        split_pair(acc[2 * kk + 1][0], acc[2 * kk + 1][1], hi[2], lo[2]);
        split_pair(acc[2 * kk + 1][2], acc[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_16816(o0[nt], hi, bh[2 * nt], bh[2 * nt + 1]);
          mma_16816(o1[nt], hi, bl[2 * nt], bl[2 * nt + 1]);
          mma_16816(o2[nt], lo, bh[2 * nt], bh[2 * nt + 1]);
        }
      }
      uint32_t bh[4], bl[4];
      const uint32_t off = (uint32_t)(nrm_row * kARow + nrm_col) * 2;
      ldsm_x4(bh, aA + off);
      ldsm_x4(bl, aAl + off);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        mma_16816(o1[nt], va, bh[2 * nt], bh[2 * nt + 1]);
        mma_16816(o2[nt], va, bl[2 * nt], bl[2 * nt + 1]);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          ob[(nt * 8 + q2 + (i & 1)) * L.obuf_row + r + (i >> 1) * 8] = o0[nt][i] + o1[nt][i] + o2[nt][i];
    } else if (warp == 0) {
#pragma unroll
      for (int k = 0; k < (dkp + 31) / 32; ++k)
        if (lane + 32 * k < dkp) whole[k] *= D[lane + 32 * k];
    }
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      uint32_t bh[4], bl[4];
      const uint32_t off = (uint32_t)(trn_row * rs + kk * 16 + trn_col) * 2;
      ldsm_x4_t(bh, akh + off);
      ldsm_x4_t(bl, akl + off);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = 2 * kk + e;
        const float2 dd = *reinterpret_cast<const float2*>(D + 8 * j + q2);
        acc[j][0] *= dd.x;
        acc[j][1] *= dd.y;
        acc[j][2] *= dd.x;
        acc[j][3] *= dd.y;
        mma_16816(acc[j], va, bh[2 * e], bh[2 * e + 1]);
        mma_16816(acc[j], va, bl[2 * e], bl[2 * e + 1]);
      }
    }
    if constexpr (OUT) {
      __syncthreads();
      const int len = min(kChunk, tokens - c * kChunk);
      const float* floor_ = D + dkp;
      const __nv_bfloat16* gt = reinterpret_cast<const __nv_bfloat16*>(st + L.g_off);
      for (int t = warp; t < len; t += n_warps) {
        const float* orow = ob + t * L.obuf_row;
        float inv = 1.f;
        if (norm) inv = 1.f / (fmaxf(fabsf(orow[p.dv]), floor_[t]) + 1e-6f);
        float2 o[kScanMaxWarps * 16 / 64];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < kScanMaxWarps * 16 / 64; ++k) {
          const int i = lane * 2 + k * 64;
          o[k] = make_float2(0.f, 0.f);
          if (i < p.dv) {
            o[k] = *reinterpret_cast<const float2*>(orow + i);
            o[k].x *= inv;
            o[k].y *= inv;
          }
          ss += o[k].x * o[k].x + o[k].y * o[k].y;
        }
        const float f = p.out_scale / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
        __nv_bfloat16* dst = out + (size_t)(c * kChunk + t) * p.out_stride;
#pragma unroll
        for (int k = 0; k < kScanMaxWarps * 16 / 64; ++k) {
          const int i = lane * 2 + k * 64;
          if (i < p.dv) {
            const float2 gv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gt + t * p.dv + i));
            const float sx = __fdividef(1.f, 1.f + __expf(-gv.x)), sy = __fdividef(1.f, 1.f + __expf(-gv.y));
            const float gx = p.gate_act == 0 ? gv.x * sx : sx, gy = p.gate_act == 0 ? gv.y * sy : sy;
            *reinterpret_cast<uint32_t*>(dst + i) = pack_bf16x2(o[k].x * f * nw[k].x * gx, o[k].y * f * nw[k].y * gy);
          }
        }
      }
    }
  }
  copy_wait<0>();
  if (OUT && !(flags & 2)) return;
  float* to = OUT ? slot_S : seg_S;
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = r + (i >> 1) * 8, d = 8 * j + q2 + (i & 1);
      if (rr < rows && d < p.dk) to[(size_t)rr * p.dk + d] = acc[j][i];
    }
  if (!OUT && warp == 0) {
#pragma unroll
    for (int k = 0; k < (dkp + 31) / 32; ++k)
      if (lane + 32 * k < dkp) sg.decay[((size_t)g_id * p.H + h) * dkp + lane + 32 * k] = whole[k];
  }
}

// start states of the segments of sequences that have several: state elements in parallel, segments in order
__global__ void segment_states_kernel(RecParams p, Segments sg, const int* __restrict__ slots,
                                      const int* __restrict__ pos0, int dkp) {
  const int h = blockIdx.y, s = blockIdx.z;
  const int rows = p.dv + (p.kind == kGateHead ? 1 : 0);
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  const int slot = slots[s], g0 = sg.seq_seg0[s], g1 = sg.seq_seg0[s + 1];
  if (e >= rows * p.dk || slot < 0 || g1 - g0 < 2) return;
  const int d = e % p.dk;
  float cur = pos0[s] == 0 ? 0.f : p.S[((size_t)slot * p.H + h) * rows * p.dk + e];
#pragma unroll 4
  for (int g = g0; g < g1; ++g) {
    float* at = sg.S + ((size_t)g * p.H + h) * rows * p.dk + e;
    float local = 0.f, decay = 0.f;
    if (g + 1 < g1) {
      local = *at;
      decay = sg.decay[((size_t)g * p.H + h) * dkp + d];
    }
    *at = cur;
    cur = fmaf(decay, cur, local);
  }
}

template <int NK>
static int launch_chunks(const RecParams& p, const Segments& sg, int n_seg, const int* slots, const int* pos0, int n_seq,
                         const int* chunk_row, const int* chunk_len, int n_chunks, const float4* gates, uint8_t* tiles,
                         cudaStream_t stream) {
  constexpr int dkp = NK * 16;
  const bool head = p.kind == kGateHead;
  const int norm = head ? 1 : 0, rows = p.dv + norm;
  const int dvp = (p.dv + norm + 15) / 16 * 16;
  const int vec = p.dk % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0;
  const size_t psm = (size_t)(3 * kChunk * (dkp + 1) + kChunk * kChunk + kChunk * 2 + (head ? 0 : kChunk * p.rank)) * 4;
  cudaError_t e;
  auto prep = head ? chunk_prepare_kernel<NK, true> : chunk_prepare_kernel<NK, false>;
  if (psm > 48 * 1024 &&
      (e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024)) != cudaSuccess)
    return (int)e;
  prep<<<dim3(n_chunks, p.H), kPrepThreads, psm, stream>>>(p, chunk_row, chunk_len, gates, tiles, vec);
  if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  const ScanSmem L(dkp, dvp, p.dv);
  static int configured = 0;
  if (configured < L.total) {
    if ((e = cudaFuncSetAttribute(chunk_scan_kernel<NK, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(chunk_scan_kernel<NK, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total)) != cudaSuccess)
      return (int)e;
    configured = L.total;
  }
  const dim3 grid(p.H, n_seg);
  const int threads = dvp / 16 * 32;
  if (n_seg > n_seq) {
    chunk_scan_kernel<NK, false><<<grid, threads, L.total, stream>>>(p, sg, slots, pos0, tiles);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    segment_states_kernel<<<dim3((rows * p.dk + 255) / 256, p.H, n_seq), 256, 0, stream>>>(p, sg, slots, pos0, dkp);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  }
  chunk_scan_kernel<NK, true><<<grid, threads, L.total, stream>>>(p, sg, slots, pos0, tiles);
  return (int)cudaGetLastError();
}

}  // namespace sb

using namespace sb;

static_assert(sizeof(RecParams) == 160, "RecParams is mirrored by a ctypes structure in ops/recurrence.py");

// One token (row0 / nrow null: row s of sequence s) or a packed portion per sequence, any sizes.  `params` is a host
// RecParams.  slots[s] < 0: idle, its output rows are zero.
extern "C" int sb_recurrence_step(const void* params, const int* row0, const int* nrow, const int* slots,
                                  const int* pos0, int n_seq, int f32, cudaStream_t stream) {
  if (n_seq == 0) return 0;
  if (n_seq > 65535) return -3;
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  const int rows = p.dv + (p.kind == kGateHead ? 1 : 0);
  const size_t base = (size_t)(3 * ((p.dk + 3) & ~3) + ((p.dv + 4) & ~3) + 8) * 4;
  const size_t state = (size_t)rows * p.dk * 4;
  const int in_smem = nrow != nullptr && base + state <= 100 * 1024;
  const size_t smem = base + (in_smem ? state : 0);
  if (base > 100 * 1024) return -3;
  const dim3 grid(p.H, n_seq);
  auto run = [&](auto kernel) -> int {
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
      if (e != cudaSuccess) return (int)e;
    }
    kernel<<<grid, kStepThreads, smem, stream>>>(p, row0, nrow, slots, pos0, in_smem);
    return (int)cudaGetLastError();
  };
  if (f32) return p.dk % 4 ? run(recurrence_step_kernel<float, 1>) : run(recurrence_step_kernel<float, 4>);
  return p.dk % 4 ? run(recurrence_step_kernel<__nv_bfloat16, 1>) : run(recurrence_step_kernel<__nv_bfloat16, 4>);
}

extern "C" int sb_recurrence_chunk() { return kChunk; }

// Bytes of workspace of sb_recurrence_prefill for `n_chunks` chunks, `n_seg` segments and `T` rows, or -1 when the sizes
// need the token-by-token kernel (dk <= 128, dv a multiple of 8, dv (+1) <= 192, 16-byte aligned rows).
extern "C" long long sb_recurrence_workspace(const void* params, int n_chunks, int n_seg, int T) {
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int dkp = (p.dk + 15) / 16 * 16, dvp = (p.dv + norm + 15) / 16 * 16;
  if (dkp > 128 || p.dv % 8 || dvp > 16 * kScanMaxWarps || p.row_stride % 8 || p.v_off % 8 || p.g_off % 8 ||
      p.out_stride % 2 || p.out_off % 2 || p.rank > 256 || ((uintptr_t)p.x & 15) || ((uintptr_t)p.out & 3) ||
      ((uintptr_t)p.norm_w & 3))
    return -1;
  return (long long)T * p.H * 16 + (long long)n_chunks * p.H * tile_bytes(dkp) +
         (long long)n_seg * p.H * 4 * ((long long)(p.dv + norm) * p.dk + dkp) + 64;
}

// bf16 prefill of packed portions in 16-token chunks: chunk c covers rows chunk_row[c] .. + chunk_len[c].  Segments are
// runs of consecutive chunks of one sequence: five int arrays of n_seg entries in `segs` (sequence, first chunk, first
// row, tokens, flags: 1 first, 2 last) and then n_seq + 1 entries with each sequence's first segment.
extern "C" int sb_recurrence_prefill(const void* params, const int* row0, const int* nrow, const int* slots,
                                     const int* pos0, int n_seq, const int* chunk_row, const int* chunk_len,
                                     int n_chunks, const int* segs, int n_seg, int T, void* workspace,
                                     cudaStream_t stream) {
  if (n_seq == 0 || n_chunks == 0) return 0;
  if (n_seq > 65535 || n_seg > 65535 || ((uintptr_t)workspace & 15)) return -3;
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  if (sb_recurrence_workspace(params, n_chunks, n_seg, T) < 0) return -2;
  const int dkp = (p.dk + 15) / 16 * 16, rows = p.dv + (p.kind == kGateHead ? 1 : 0);
  float4* gates = reinterpret_cast<float4*>(workspace);
  uint8_t* tiles = reinterpret_cast<uint8_t*>(workspace) + (size_t)T * p.H * 16;
  Segments sg;
  sg.seq = segs; sg.chunk0 = segs + n_seg; sg.row = segs + 2 * n_seg; sg.tokens = segs + 3 * n_seg;
  sg.flags = segs + 4 * n_seg; sg.seq_seg0 = segs + 5 * n_seg;
  sg.S = reinterpret_cast<float*>(tiles + (size_t)n_chunks * p.H * tile_bytes(dkp));
  sg.decay = sg.S + (size_t)n_seg * p.H * rows * p.dk;
  if (p.kind == kGateHead) {
    gate_scan_kernel<<<dim3(p.H, n_seq), kGsThreads, 0, stream>>>(p, row0, nrow, slots, pos0, gates);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
  }
  switch (dkp / 16) {
#define SB_SCAN(NK) \
  case NK:          \
    return launch_chunks<NK>(p, sg, n_seg, slots, pos0, n_seq, chunk_row, chunk_len, n_chunks, gates, tiles, stream);
    SB_SCAN(1) SB_SCAN(2) SB_SCAN(3) SB_SCAN(4) SB_SCAN(5) SB_SCAN(6) SB_SCAN(7) SB_SCAN(8)
#undef SB_SCAN
  }
  return -2;
}
