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
//   chunk_prepare_kernel     prefill, kGateChannel: everything of a 16-token chunk that does not depend on the state, in
//                            parallel over chunks and heads: q and k scaled by their decays to the chunk's start / end, the 16 x 16
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
#include "recurrence.cuh"

namespace sb {

__device__ __forceinline__ float log_sigmoid(float x) {
  return x >= 0.f ? -log1pf(expf(-x)) : x - log1pf(expf(x));
}
// base 2, error of a few 1e-7 absolute: that of a sigmoid rounded to fp32
__device__ __forceinline__ float log2_sigmoid(float x) {
  return fminf(x, 0.f) * 1.4426950408889634f - log2f(1.f + __expf(-fabsf(x)));
}
template <typename T>
__device__ __forceinline__ void head_gates(const RecParams& p, const T* xr, int h, float& i, float& f) {
  const float zi = to_float(xr[p.e_off + h]) + to_float(reinterpret_cast<const T*>(p.b_e)[h]);
  const float zf = to_float(xr[p.f_off + h]) + to_float(reinterpret_cast<const T*>(p.b_f)[h]);
  i = p.cap * tanhf(zi / p.cap);
  f = log_sigmoid(p.cap * tanhf(zf / p.cap));
}

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
constexpr int kGsThreads = 512, kGsPer = 8;

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
__host__ __device__ inline int tile_bytes(int dkp) {
  return 4 * kChunk * tile_row(dkp) * 2 + 2 * kChunk * kARow * 2 + dkp * 4;
}

constexpr int kPrepThreads = 128;

// kGateChannel only; NK: key channels in steps of 16 (padded)
template <int NK>
__global__ void __launch_bounds__(kPrepThreads)
chunk_prepare_kernel(RecParams p, const int* __restrict__ chunk_row, const int* __restrict__ chunk_len,
                     uint8_t* __restrict__ tiles, int vec) {
  constexpr int dkp = NK * 16, ld = dkp + 1, rs = dkp + 8;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                       // [16][ld]
  float* sk = sq + kChunk * ld;
  float* sc = sk + kChunk * ld;         // log2 of the decay from the chunk's start through token t
  float* sA = sc + kChunk * ld;         // [16][16], 16-byte aligned (16 ld floats are a multiple of four)
  float* se = sA + kChunk * kChunk;     // low-rank rows [16][rank]
  const bool w_vec = p.rank % 8 == 0 && ((uintptr_t)p.w2 & 15) == 0;
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
  for (int i = tid; i < kChunk * p.rank; i += kPrepThreads) {
    const int t = i / p.rank;
    const int r = i - t * p.rank;
    se[r * kChunk + t] = t < len ? to_float(x[(size_t)t * p.row_stride + p.e_off + r]) : 0.f;
  }
  __syncthreads();
  // log decays of (channel, group of 8 tokens) items, then running sums per channel
  for (int i = tid; i < dkp * 2; i += kPrepThreads) {
    const int d = i % dkp, t0 = i / dkp * 8;
    const bool ok = d < p.dk;
    const float b = ok ? to_float(reinterpret_cast<const __nv_bfloat16*>(p.b_e)[h * p.dk + d]) : 0.f;
    float z[8];
#pragma unroll
    for (int t = 0; t < 8; ++t) z[t] = b;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w2) + (size_t)(h * p.dk + (ok ? d : 0)) * p.rank;
    auto step = [&](float wr, int r) {
      const float4 a = *reinterpret_cast<const float4*>(se + r * kChunk + t0), b4 = *reinterpret_cast<const float4*>(se + r * kChunk + t0 + 4);
      z[0] = fmaf(wr, a.x, z[0]);
      z[1] = fmaf(wr, a.y, z[1]);
      z[2] = fmaf(wr, a.z, z[2]);
      z[3] = fmaf(wr, a.w, z[3]);
      z[4] = fmaf(wr, b4.x, z[4]);
      z[5] = fmaf(wr, b4.y, z[5]);
      z[6] = fmaf(wr, b4.z, z[6]);
      z[7] = fmaf(wr, b4.w, z[7]);
    };
    if (w_vec) {
      for (int r0 = 0; r0 < p.rank; r0 += 8) {
        float wr[8];
        load_vec<__nv_bfloat16, 8>(w + r0, wr);
#pragma unroll
        for (int r = 0; r < 8; ++r) step(wr[r], r0 + r);
      }
    } else {
      for (int r = 0; r < p.rank; ++r) step(to_float(w[r]), r);
    }
#pragma unroll
    for (int t = 0; t < 8; ++t)
      sc[(t0 + t) * ld + d] = (t0 + t < len && ok) ? log2_sigmoid(z[t]) * p.inv_tau : 0.f;
  }
  __syncthreads();
  for (int d = tid; d < dkp; d += kPrepThreads) {
    float acc = 0.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      acc += sc[t * ld + d];
      sc[t * ld + d] = acc;
    }
    D[d] = ex2(acc);
  }
  __syncthreads();
  // decayed q (to the chunk's start) and k (to its end)
  for (int i = tid; i < kChunk * (dkp / 2); i += kPrepThreads) {
    const int t = i / (dkp / 2), d = i % (dkp / 2) * 2;
    const float c0 = sc[t * ld + d], c1 = sc[t * ld + d + 1];
    const float e0 = sc[(kChunk - 1) * ld + d], e1 = sc[(kChunk - 1) * ld + d + 1];
    uint32_t hi, lo;
    split_pair(sq[t * ld + d] * ex2(c0), sq[t * ld + d + 1] * ex2(c1), hi, lo);
    *reinterpret_cast<uint32_t*>(qh + t * rs + d) = hi;
    *reinterpret_cast<uint32_t*>(ql + t * rs + d) = lo;
    split_pair(sk[t * ld + d] * ex2(e0 - c0), sk[t * ld + d + 1] * ex2(e1 - c1), hi, lo);
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
        ct[i] = sc[(bi * 4 + i) * ld + d];
        cs[i] = sc[(bj * 4 + i) * ld + d];
      }
      if (bi > bj) {
        const float anchor = sc[(bi * 4 - 1) * ld + d];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          q[i] *= ex2(ct[i] - anchor);
          k[i] *= ex2(anchor - cs[i]);
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) a[i] = fmaf(q[i / 4], k[i % 4], a[i]);
      } else {
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (i % 4 <= i / 4) a[i] = fmaf(q[i / 4] * k[i % 4], i / 4 == i % 4 ? 1.f : ex2(ct[i / 4] - cs[i % 4]), a[i]);
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
    if (!(lane & 1) && s <= t) sA[t * kChunk + s] = v;
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
constexpr int kScanMaxWarps = 12;
constexpr int kScanStages = 3;

// threads of a block and blocks that fit an SM (registers)
__host__ __device__ constexpr int scan_threads(int dv, bool scalar) { return 32 * (dv / 16 + (scalar && dv == 128 ? 1 : 0)); }
__host__ __device__ constexpr int scan_blocks(int nk, int dv) { return nk > 4 || dv > 128 ? 1 : 2; }

// shared memory of the scan: stages of {q / k material, value rows, gates}, then two output buffers
template <bool SCALAR>
struct ScanSmem {
  int tile, v_row, v_off, gate_off, stage, obuf_off, obuf_row, obuf, norm_off, total;
  __host__ __device__ ScanSmem(int dkp, int dvp) {
    tile = SCALAR ? 2 * kChunk * tile_row(dkp) * 2 : tile_bytes(dkp);
    v_row = dvp + 8;
    v_off = tile;
    gate_off = v_off + kChunk * v_row * 2;
    stage = (gate_off + (SCALAR ? kChunk * 16 : 0) + 127) / 128 * 128;
    obuf_off = kScanStages * stage;
    obuf_row = dvp + 4;
    obuf = kChunk * obuf_row;
    norm_off = obuf_off + 2 * obuf * 4;
    total = norm_off + dvp * 4;
  }
};

// Warp w of the CTA owns value columns 16 w .. 16 w + 15 (rows of the fragments) and all key channels (NK steps of 16).
// Iteration c multiplies chunk c and finishes (norm, gate, store) chunk c - 1: one block barrier per chunk.
//
// SCALAR (one decay per head and token): q, k and v arrive as projected.  Decays and write weights multiply the fp32
// results (rows of o), the score fragments and the value fragments, so q and k enter the products exactly.
template <int NK, int DV, bool SCALAR, bool OUT>
__global__ void __launch_bounds__(scan_threads(DV, SCALAR), scan_blocks(NK, DV))
chunk_scan_kernel(RecParams p, Segments sg, const int* __restrict__ slots, const int* __restrict__ pos0,
                  const uint8_t* __restrict__ tiles, const float4* __restrict__ gates) {
  constexpr int dkp = NK * 16, rs = dkp + 8, KD = DV / 64;
  constexpr int kStateOff = SCALAR ? kChunk * rs * 2 : 2 * kChunk * rs * 2;           // keys of the state update
  constexpr int kDOff = 4 * kChunk * rs * 2 + 2 * kChunk * kARow * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int norm = SCALAR ? 1 : 0;
  const int dvp = (p.dv + norm + 15) / 16 * 16;
  const ScanSmem<SCALAR> L(dkp, dvp);
  float* obuf = reinterpret_cast<float*>(smem + L.obuf_off);
  const int h = blockIdx.x, g_id = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_warps = blockDim.x >> 5;
  const int s = sg.seq[g_id], slot = slots[s], flags = sg.flags[g_id];
  if (slot < 0 || (!OUT && (flags & 2))) return;
  const int tokens = sg.tokens[g_id], n = (tokens + kChunk - 1) / kChunk, row0 = sg.row[g_id];
  const uint8_t* my_tiles = SCALAR ? nullptr : tiles + ((size_t)sg.chunk0[g_id] * p.H + h) * L.tile;
  const size_t tile_step = (size_t)p.H * L.tile;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)row0 * p.row_stride;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)row0 * p.out_stride + p.out_off + (size_t)h * p.dv;

  // parts of the stages that no copy writes: zeros, and ones for the normaliser's value column
  for (int st = 0; st < kScanStages; ++st) {
    uint8_t* base = smem + st * L.stage;
    __nv_bfloat16* v = reinterpret_cast<__nv_bfloat16*>(base + L.v_off);
    const int extra = L.v_row - p.dv;
    for (int i = tid; i < kChunk * extra; i += blockDim.x)
      v[i / extra * L.v_row + p.dv + i % extra] = __float2bfloat16(norm && i % extra == 0 ? 1.f : 0.f);
    if constexpr (SCALAR)
      for (int i = tid; i < 2 * kChunk * (rs - p.dk); i += blockDim.x)
        reinterpret_cast<__nv_bfloat16*>(base)[i / (rs - p.dk) * rs + p.dk + i % (rs - p.dk)] = __float2bfloat16(0.f);
  }
  // copies of `width` (a multiple of 8) bf16 columns of the chunk's rows into a tile with row pitch `pitch`; the place
  // of a thread's first vector does not change from chunk to chunk
  const int v_t = tid / (p.dv / 8), v_e = (tid - v_t * (p.dv / 8)) * 8, k_t = SCALAR ? tid / (p.dk / 8) : 0,
            k_e = SCALAR ? (tid - k_t * (p.dk / 8)) * 8 : 0;
  auto copy_rows = [&](uint8_t* dst, int pitch, const __nv_bfloat16* src, int width, int len, int t, int e) {
    if (t < kChunk) {
      if (t < len) copy16(dst + (t * pitch + e) * 2, src + t * p.row_stride + e);
      else *reinterpret_cast<uint4*>(dst + (t * pitch + e) * 2) = make_uint4(0, 0, 0, 0);
    }
    const int nv = width / 8;
    for (int i = tid + blockDim.x; i < kChunk * nv; i += blockDim.x) {
      const int t2 = i / nv, e2 = (i - t2 * nv) * 8;
      if (t2 < len) copy16(dst + (t2 * pitch + e2) * 2, src + t2 * p.row_stride + e2);
      else *reinterpret_cast<uint4*>(dst + (t2 * pitch + e2) * 2) = make_uint4(0, 0, 0, 0);
    }
  };
  auto issue = [&](int c) {      // copies of chunk c into its stage (an empty group past the end)
    if (c < n) {
      uint8_t* st = smem + (c % kScanStages) * L.stage;
      const int len = min(kChunk, tokens - c * kChunk);
      const __nv_bfloat16* xc = x + (size_t)c * kChunk * p.row_stride;
      if constexpr (SCALAR) {
        if (OUT) copy_rows(st, rs, xc + p.q_off + h * p.dk, p.dk, len, k_t, k_e);
        copy_rows(st + kStateOff, rs, xc + p.k_off + h * p.dk, p.dk, len, k_t, k_e);
        if (tid < kChunk) {
          uint8_t* dst = st + L.gate_off + tid * 16;
          if (tid < len) copy16(dst, gates + (size_t)(row0 + c * kChunk + tid) * p.H + h);
          else *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 1.f, 0.f);
        }
      } else {
        const uint8_t* src = my_tiles + (size_t)c * tile_step;
        for (int i = tid * 16 + (OUT ? 0 : kStateOff); i < L.tile; i += blockDim.x * 16) copy16(st + i, src + i);
      }
      copy_rows(st + L.v_off, L.v_row, xc + p.v_off + h * p.dv, p.dv, len, v_t, v_e);
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
  float* nw = reinterpret_cast<float*>(smem + L.norm_off);
  if (OUT)
    for (int i = tid; i < p.dv; i += blockDim.x)
      nw[i] = to_float(reinterpret_cast<const __nv_bfloat16*>(p.norm_w)[(p.norm_per_head ? h * p.dv : 0) + i]);
  float whole[SCALAR ? 1 : (dkp + 31) / 32];            // pass 0: product of the chunks' decays
#pragma unroll
  for (float& w : whole) w = 1.f;
  const float inv_dv = 1.f / (float)p.dv;
  float floor_t = 1.f;                                  // SCALAR: lane t holds exp(-m_t) of the chunk to be finished

  // lane's row / column offsets inside a 16 x 16 tile for the two ldmatrix arrangements
  const int nrm_row = (lane & 7) + ((lane >> 4) << 3), nrm_col = ((lane >> 3) & 1) * 8;   // rows 0-7: columns 0-7, 8-15
  const int trn_row = (lane & 7) + (((lane >> 3) & 1) << 3), trn_col = (lane >> 4) * 8;   // columns 0-7: rows 0-7, 8-15

  for (int c = 0; c <= n; ++c) {
    if (c < n) copy_wait<kScanStages - 2>();
    else if (!OUT) break;
    __syncthreads();            // chunk c has landed, chunk c - 1 is multiplied, chunk c - 2 is out
    issue(c + kScanStages - 1);
    // each half warp finishes one token: four values per lane and 64 columns
    const int et = (c - 1) * kChunk + warp * 2 + (lane >> 4);
    uint2 gpre[KD];             // output-gate values of chunk c - 1, fetched ahead of their use
    if constexpr (OUT) {
#pragma unroll
      for (int k = 0; k < KD; ++k) {
        const int i = (lane & 15) * 4 + k * 64;
        gpre[k] = make_uint2(0, 0);
        if (c > 0 && warp * 2 < kChunk && et < tokens && i < p.dv)
          gpre[k] = *reinterpret_cast<const uint2*>(x + (size_t)et * p.row_stride + p.g_off + h * p.dv + i);
      }
    }
    const float floor_prev = floor_t;
    if (c < n) {
      const uint8_t* st = smem + (c % kScanStages) * L.stage;
      const uint32_t a_q = smem_u32(st), a_k = a_q + kStateOff;
      uint32_t va[4];             // v^T: value columns x tokens
      ldsm_x4_t(va, smem_u32(st + L.v_off) + (uint32_t)(nrm_row * L.v_row + warp * 16 + nrm_col) * 2);
      float* ob = obuf + (c & 1) * L.obuf;
      if constexpr (SCALAR) {
        // lane t: decay from the chunk's start through token t, write weight (both log 2)
        const float4 gt = *reinterpret_cast<const float4*>(st + L.gate_off + (lane & 15) * 16);
        float ct = gt.x * kLog2e;
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) {
          const float up = __shfl_up_sync(0xffffffffu, ct, o);
          if ((lane & 15) >= o) ct += up;
        }
        const float lw = gt.y * kLog2e;
        const float ce = __shfl_sync(0xffffffffu, ct, 15);
        floor_t = gt.z;
        const float whole_c = ex2(ce);
        const float put_s = ex2(ce - ct + lw);           // of lane t's token: weight in the chunk's end state
        if constexpr (OUT) {
          float o0[2][4] = {}, o1[2][4] = {}, pr[2][4] = {};
#pragma unroll
          for (int kk = 0; kk < NK; ++kk) {
            uint32_t qf[4], kf[4], hi[4], lo[4];
            ldsm_x4(qf, a_q + (uint32_t)(trn_row * rs + kk * 16 + trn_col) * 2);
            ldsm_x4(kf, a_k + (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2);
            split_pair(acc[2 * kk][0], acc[2 * kk][1], hi[0], lo[0]);
            split_pair(acc[2 * kk][2], acc[2 * kk][3], hi[1], lo[1]);
            split_pair(acc[2 * kk + 1][0], acc[2 * kk + 1][1], hi[2], lo[2]);
            split_pair(acc[2 * kk + 1][2], acc[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
              mma_16816(o0[nt], hi, qf[nt], qf[nt + 2]);
              mma_16816(o1[nt], lo, qf[nt], qf[nt + 2]);
              mma_16816(pr[nt], qf, kf[2 * nt], kf[2 * nt + 1]);
            }
          }
          // pr[nt]: scores of rows t = g, g + 8 with s = 8 nt + 2 (lane % 4) + {0, 1}; decayed, they are the second
          // operand of o^T += v^T P^T as they lie
          const float c_lo = __shfl_sync(0xffffffffu, ct, g), c_hi = __shfl_sync(0xffffffffu, ct, g + 8);
          uint32_t ph[2][2], pl[2][2];      // [t half][s half]
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int s0 = nt * 8 + q2;
            const float e0 = __shfl_sync(0xffffffffu, lw - ct, s0), e1 = __shfl_sync(0xffffffffu, lw - ct, s0 + 1);
            const float a0 = s0 <= g ? pr[nt][0] * p.q_scale * ex2(c_lo + e0) : 0.f;
            const float a1 = s0 + 1 <= g ? pr[nt][1] * p.q_scale * ex2(c_lo + e1) : 0.f;
            const float a2 = s0 <= g + 8 ? pr[nt][2] * p.q_scale * ex2(c_hi + e0) : 0.f;
            const float a3 = s0 + 1 <= g + 8 ? pr[nt][3] * p.q_scale * ex2(c_hi + e1) : 0.f;
            split_pair(a0, a1, ph[0][nt], pl[0][nt]);
            split_pair(a2, a3, ph[1][nt], pl[1][nt]);
          }
          const float fo = ex2(ct) * p.q_scale;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const float f0 = __shfl_sync(0xffffffffu, fo, nt * 8 + q2), f1 = __shfl_sync(0xffffffffu, fo, nt * 8 + q2 + 1);
            float o[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) o[i] = (o0[nt][i] + o1[nt][i]) * (i & 1 ? f1 : f0);
            mma_16816(o, va, ph[nt][0], ph[nt][1]);
            mma_16816(o, va, pl[nt][0], pl[nt][1]);
#pragma unroll
            for (int i = 0; i < 4; ++i) ob[(nt * 8 + q2 + (i & 1)) * L.obuf_row + r + (i >> 1) * 8] = o[i];
          }
        } else {
          whole[0] *= whole_c;
        }
        // values with their weights, in two terms
        uint32_t vh[4], vl[4];
#pragma unroll
        for (int sh = 0; sh < 2; ++sh) {
          const float w0 = __shfl_sync(0xffffffffu, put_s, sh * 8 + q2), w1 = __shfl_sync(0xffffffffu, put_s, sh * 8 + q2 + 1);
#pragma unroll
          for (int b = 0; b < 2; ++b) {
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&va[sh * 2 + b]));
            split_pair(v.x * w0, v.y * w1, vh[sh * 2 + b], vl[sh * 2 + b]);
          }
        }
#pragma unroll
        for (int kk = 0; kk < NK; ++kk) {
          uint32_t kf[4];
          ldsm_x4_t(kf, a_k + (uint32_t)(trn_row * rs + kk * 16 + trn_col) * 2);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[2 * kk + e][i] *= whole_c;
            mma_16816(acc[2 * kk + e], vh, kf[2 * e], kf[2 * e + 1]);
            mma_16816(acc[2 * kk + e], vl, kf[2 * e], kf[2 * e + 1]);
          }
        }
      } else {
        const uint32_t a_ql = a_q + kChunk * rs * 2, a_kl = a_k + kChunk * rs * 2;
        const float* D = reinterpret_cast<const float*>(st + kDOff);
        if constexpr (OUT) {
          const uint32_t aA = a_kl + kChunk * rs * 2, aAl = aA + kChunk * kARow * 2;
          float o0[2][4] = {}, o1[2][4] = {}, o2[2][4] = {};
#pragma unroll
          for (int kk = 0; kk < NK; ++kk) {
            uint32_t hi[4], lo[4], bh[4], bl[4];
            const uint32_t off = (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2;
            ldsm_x4(bh, a_q + off);
            ldsm_x4(bl, a_ql + off);
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
          ldsm_x4_t(bh, a_k + off);
          ldsm_x4_t(bl, a_kl + off);
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
      }
    }
    if constexpr (OUT) {
      if (c == 0) continue;
      const float* ob = obuf + ((c - 1) & 1) * L.obuf;
      const int t0 = (c - 1) * kChunk, len = min(kChunk, tokens - t0);
      for (int tb = warp * 2; tb < len; tb += n_warps * 2) {
        const int t = tb + (lane >> 4);                    // below 16; rows past `len` are computed and not stored
        const float* orow = ob + t * L.obuf_row;
        float inv = 1.f;
        if constexpr (SCALAR)
          inv = __fdividef(1.f, fmaxf(fabsf(orow[p.dv]), __shfl_sync(0xffffffffu, floor_prev, t)) + 1e-6f);
        float4 o[KD];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < KD; ++k) {
          const int i = (lane & 15) * 4 + k * 64;
          o[k] = i < p.dv ? *reinterpret_cast<const float4*>(orow + i) : make_float4(0.f, 0.f, 0.f, 0.f);
          o[k].x *= inv;
          o[k].y *= inv;
          o[k].z *= inv;
          o[k].w *= inv;
          ss += o[k].x * o[k].x + o[k].y * o[k].y + o[k].z * o[k].z + o[k].w * o[k].w;
        }
#pragma unroll
        for (int w = 8; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
        const float f = p.out_scale * rsqrtf(ss * inv_dv + p.eps);
        if (t < len) {
          __nv_bfloat16* dst = out + (size_t)(t0 + t) * p.out_stride;
#pragma unroll
          for (int k = 0; k < KD; ++k) {
            const int i = (lane & 15) * 4 + k * 64;
            if (i < p.dv) {
              const uint2 graw = tb == warp * 2 ? gpre[k] : *reinterpret_cast<const uint2*>(
                                     x + (size_t)(t0 + t) * p.row_stride + p.g_off + h * p.dv + i);
              const float4 w = *reinterpret_cast<const float4*>(nw + i);
              const float2 ga = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&graw.x));
              const float2 gb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&graw.y));
              uint2 y;
              y.x = pack_bf16x2(o[k].x * f * w.x * fast_gate(ga.x, p.gate_act), o[k].y * f * w.y * fast_gate(ga.y, p.gate_act));
              y.y = pack_bf16x2(o[k].z * f * w.z * fast_gate(gb.x, p.gate_act), o[k].w * f * w.w * fast_gate(gb.y, p.gate_act));
              *reinterpret_cast<uint2*>(dst + i) = y;
            }
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
      if (lane + 32 * k < dkp) sg.decay[((size_t)g_id * p.H + h) * dkp + lane + 32 * k] = whole[SCALAR ? 0 : k];
  }
}

// start states of the segments of sequences that have several: state elements in parallel, segments in order (eight
// local states are fetched ahead of the stores that replace them)
__global__ void segment_states_kernel(RecParams p, Segments sg, const int* __restrict__ slots,
                                      const int* __restrict__ pos0, int dkp) {
  const int h = blockIdx.y, s = blockIdx.z;
  const int rows = p.dv + (p.kind == kGateHead ? 1 : 0);
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  const int slot = slots[s], g0 = sg.seq_seg0[s], g1 = sg.seq_seg0[s + 1];
  if (e >= rows * p.dk || slot < 0 || g1 - g0 < 2) return;
  const int d = e % p.dk;
  const size_t step = (size_t)p.H * rows * p.dk;
  float* at = sg.S + ((size_t)g0 * p.H + h) * rows * p.dk + e;
  const float* dec = sg.decay + ((size_t)g0 * p.H + h) * dkp + d;
  float cur = pos0[s] == 0 ? 0.f : p.S[((size_t)slot * p.H + h) * rows * p.dk + e];
  for (int b = 0; b < g1 - g0; b += 8) {
    float local[8], decay[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const bool has = b + k + 1 < g1 - g0;      // the last segment leaves no local state
      local[k] = has ? at[(size_t)(b + k) * step] : 0.f;
      decay[k] = has ? dec[(size_t)(b + k) * p.H * dkp] : 0.f;
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      if (b + k < g1 - g0) at[(size_t)(b + k) * step] = cur;
      cur = fmaf(decay[k], cur, local[k]);
    }
  }
}

template <int NK, int DV, bool SCALAR>
static int launch_scans(const RecParams& p, const Segments& sg, int n_seg, const int* slots, const int* pos0, int n_seq,
                        const float4* gates, const uint8_t* tiles, cudaStream_t stream) {
  constexpr int dkp = NK * 16;
  const int rows = p.dv + SCALAR, dvp = (rows + 15) / 16 * 16;
  const ScanSmem<SCALAR> L(dkp, dvp);
  cudaError_t e;
  static int configured = 0;
  if (configured < L.total) {
    if ((e = cudaFuncSetAttribute(chunk_scan_kernel<NK, DV, SCALAR, false>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                  L.total)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(chunk_scan_kernel<NK, DV, SCALAR, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                  L.total)) != cudaSuccess)
      return (int)e;
    configured = L.total;
  }
  const dim3 grid(p.H, n_seg);
  const int threads = dvp / 16 * 32;
  if (n_seg > n_seq) {
    chunk_scan_kernel<NK, DV, SCALAR, false><<<grid, threads, L.total, stream>>>(p, sg, slots, pos0, tiles, gates);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    segment_states_kernel<<<dim3((rows * p.dk + 255) / 256, p.H, n_seq), 256, 0, stream>>>(p, sg, slots, pos0, dkp);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  }
  chunk_scan_kernel<NK, DV, SCALAR, true><<<grid, threads, L.total, stream>>>(p, sg, slots, pos0, tiles, gates);
  return (int)cudaGetLastError();
}

template <int NK>
static int launch_chunks(const RecParams& p, const Segments& sg, int n_seg, const int* slots, const int* pos0, int n_seq,
                         const int* chunk_row, const int* chunk_len, int n_chunks, const float4* gates, uint8_t* tiles,
                         cudaStream_t stream) {
  if (p.kind == kGateHead)
    return p.dv <= 128 ? launch_scans<NK, 128, true>(p, sg, n_seg, slots, pos0, n_seq, gates, tiles, stream)
                       : launch_scans<NK, 192, true>(p, sg, n_seg, slots, pos0, n_seq, gates, tiles, stream);
  constexpr int dkp = NK * 16;
  const int vec = p.dk % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0;
  const size_t psm = (size_t)(3 * kChunk * (dkp + 1) + kChunk * kChunk + kChunk * p.rank) * 4;
  cudaError_t e;
  if (psm > 48 * 1024 && (e = cudaFuncSetAttribute(chunk_prepare_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                   64 * 1024)) != cudaSuccess)
    return (int)e;
  chunk_prepare_kernel<NK><<<dim3(n_chunks, p.H), kPrepThreads, psm, stream>>>(p, chunk_row, chunk_len, tiles, vec);
  if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  return p.dv <= 128 ? launch_scans<NK, 128, false>(p, sg, n_seg, slots, pos0, n_seq, gates, tiles, stream)
                     : launch_scans<NK, 192, false>(p, sg, n_seg, slots, pos0, n_seq, gates, tiles, stream);
}

}  // namespace sb

using namespace sb;

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

// (segment, head) blocks of the chunk scan that run at a time on the whole GPU
extern "C" int sb_recurrence_resident(const void* params) {
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  return num_sms() * scan_blocks(pad_dk(p.dk) / 16, p.dv <= 128 ? 128 : 192);
}

// Bytes of workspace of sb_recurrence_prefill for `n_chunks` chunks, `n_seg` segments and `T` rows, or -1 when the sizes
// need the token-by-token kernel (dk <= 128, dv a multiple of 8, dv (+1) <= 192, 16-byte aligned rows; the head form also dk a multiple of 8).
extern "C" long long sb_recurrence_workspace(const void* params, int n_chunks, int n_seg, int T) {
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int dkp = pad_dk(p.dk), dvp = (p.dv + norm + 15) / 16 * 16;
  if (norm && (p.dk % 8 || p.q_off % 8 || p.k_off % 8)) return -1;
  if (dkp > 128 || p.dv % 8 || dvp > 16 * kScanMaxWarps || p.row_stride % 8 || p.v_off % 8 ||
      p.g_off % 4 || p.out_stride % 4 || p.out_off % 4 || p.rank > 256 || ((uintptr_t)p.x & 15) || ((uintptr_t)p.out & 7))
    return -1;
  return (long long)T * p.H * 16 + (norm ? 0 : (long long)n_chunks * p.H * tile_bytes(dkp)) +
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
  const int dkp = pad_dk(p.dk), rows = p.dv + (p.kind == kGateHead ? 1 : 0);
  float4* gates = reinterpret_cast<float4*>(workspace);
  uint8_t* tiles = reinterpret_cast<uint8_t*>(workspace) + (size_t)T * p.H * 16;
  Segments sg;
  sg.seq = segs; sg.chunk0 = segs + n_seg; sg.row = segs + 2 * n_seg; sg.tokens = segs + 3 * n_seg;
  sg.flags = segs + 4 * n_seg; sg.seq_seg0 = segs + 5 * n_seg;
  sg.S = reinterpret_cast<float*>(tiles + (p.kind == kGateHead ? 0 : (size_t)n_chunks * p.H * tile_bytes(dkp)));
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
    SB_SCAN(1) SB_SCAN(2) SB_SCAN(3) SB_SCAN(4) SB_SCAN(6) SB_SCAN(8)
#undef SB_SCAN
  }
  return -2;
}
