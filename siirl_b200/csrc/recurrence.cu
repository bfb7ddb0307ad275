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
//   chunk_scan_kernel        prefill: walks the chunks of one (sequence, head) with the state in registers as tensor-core
//                            fragments; tiles arrive through a ring of bulk asynchronous copies
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

__device__ __forceinline__ void split_store(__nv_bfloat16* hi, __nv_bfloat16* lo, float x) {
  const __nv_bfloat16 a = __float2bfloat16(x);
  *hi = a;
  *lo = __float2bfloat16(x - __bfloat162float(a));
}

constexpr int kPrepThreads = 128;

__global__ void __launch_bounds__(kPrepThreads)
chunk_prepare_kernel(RecParams p, const int* __restrict__ chunk_row, const int* __restrict__ chunk_len,
                     const float4* __restrict__ gates, uint8_t* __restrict__ tiles, int dkp) {
  extern __shared__ __align__(16) float sm[];
  const int ld = dkp + 1;
  float* sq = sm;                       // [16][ld]
  float* sk = sq + kChunk * ld;
  float* sc = sk + kChunk * ld;         // log2 of the decay from the chunk's start through token t
  float* sA = sc + kChunk * ld;         // [16][16]
  float* se = sA + kChunk * kChunk;     // low-rank rows [16][rank] (kGateChannel)
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row = chunk_row[c], len = chunk_len[c];
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)row * p.row_stride;
  uint8_t* tile = tiles + ((size_t)c * p.H + h) * tile_bytes(dkp);
  const int rs = tile_row(dkp);
  __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(tile);
  __nv_bfloat16* ql = qh + kChunk * rs;
  __nv_bfloat16* kh = ql + kChunk * rs;
  __nv_bfloat16* kl = kh + kChunk * rs;
  __nv_bfloat16* Ah = kl + kChunk * rs;
  __nv_bfloat16* Al = Ah + kChunk * kARow;
  float* D = reinterpret_cast<float*>(Al + kChunk * kARow);
  float* floor_ = D + dkp;
  const bool scalar = p.kind == kGateHead;

  for (int i = tid; i < kChunk * kChunk; i += kPrepThreads) sA[i] = 0.f;
  for (int i = tid; i < kChunk * dkp; i += kPrepThreads) {
    const int t = i / dkp, d = i % dkp;
    float q = 0.f, k = 0.f;
    if (t < len && d < p.dk) {
      const __nv_bfloat16* xr = x + (size_t)t * p.row_stride;
      q = to_float(xr[p.q_off + h * p.dk + d]) * p.q_scale;
      k = to_float(xr[p.k_off + h * p.dk + d]);
      if (scalar) k *= expf(gates[(size_t)(row + t) * p.H + h].y);
    }
    sq[t * ld + d] = q;
    sk[t * ld + d] = k;
  }
  if (!scalar)
    for (int i = tid; i < kChunk * p.rank; i += kPrepThreads) {
      const int t = i / p.rank;
      se[i] = t < len ? to_float(x[(size_t)t * p.row_stride + p.e_off + i % p.rank]) : 0.f;
    }
  __syncthreads();
  for (int d = tid; d < dkp; d += kPrepThreads) {
    float acc = 0.f;
    if (scalar) {
      for (int t = 0; t < kChunk; ++t) {
        if (t < len) acc += gates[(size_t)(row + t) * p.H + h].x * kLog2e;
        sc[t * ld + d] = acc;
      }
    } else {
      float z[kChunk];
      const bool ok = d < p.dk;
      const float b = ok ? to_float(reinterpret_cast<const __nv_bfloat16*>(p.b_e)[h * p.dk + d]) : 0.f;
#pragma unroll
      for (int t = 0; t < kChunk; ++t) z[t] = b;
      const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w2) + (size_t)(h * p.dk + (ok ? d : 0)) * p.rank;
      for (int r = 0; r < p.rank; ++r) {
        const float wr = to_float(w[r]);
#pragma unroll
        for (int t = 0; t < kChunk; ++t) z[t] = fmaf(wr, se[t * p.rank + r], z[t]);
      }
#pragma unroll
      for (int t = 0; t < kChunk; ++t) {
        if (t < len && ok) acc += log_sigmoid(z[t]) * p.inv_tau * kLog2e;
        sc[t * ld + d] = acc;
      }
    }
    D[d] = exp2f(acc);
  }
  __syncthreads();
  // decayed q (to the chunk's start) and k (to its end)
  for (int i = tid; i < kChunk * dkp; i += kPrepThreads) {
    const int t = i / dkp, d = i % dkp;
    const float ct = sc[t * ld + d], ce = sc[(kChunk - 1) * ld + d];
    split_store(qh + t * rs + d, ql + t * rs + d, sq[t * ld + d] * exp2f(ct));
    split_store(kh + t * rs + d, kl + t * rs + d, sk[t * ld + d] * exp2f(ce - ct));
  }
  // scores of the chunk with itself: 4 x 4 blocks of (t, s), lanes over the key channels.  Below the diagonal the decay
  // is split at the token before the block's rows, so both factors are at most one.
  for (int blk = warp; blk < 10; blk += kPrepThreads / 32) {
    int bi = 0, bj = blk;
    while (bj > bi) {
      bj -= bi + 1;
      ++bi;
    }
    float a[4][4] = {};
    for (int d = lane; d < p.dk; d += 32) {
      float q[4], k[4], ct[4], cs[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        q[i] = sq[(bi * 4 + i) * ld + d];
        ct[i] = sc[(bi * 4 + i) * ld + d];
        k[i] = sk[(bj * 4 + i) * ld + d];
        cs[i] = sc[(bj * 4 + i) * ld + d];
      }
      if (scalar) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) a[i][j] = fmaf(q[i], k[j], a[i][j]);
      } else if (bi > bj) {
        const float anchor = sc[(bi * 4 - 1) * ld + d];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          q[i] *= exp2f(ct[i] - anchor);
          k[i] *= exp2f(anchor - cs[i]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) a[i][j] = fmaf(q[i], k[j], a[i][j]);
      } else {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j <= i; ++j) a[i][j] = fmaf(q[i] * k[j], i == j ? 1.f : exp2f(ct[i] - cs[j]), a[i][j]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float v = warp_sum(a[i][j]);
        if (lane == i * 4 + j) {
          const int t = bi * 4 + i, s = bj * 4 + j;
          if (s <= t) sA[t * kChunk + s] = scalar ? v * exp2f(sc[t * ld] - sc[s * ld]) : v;
        }
      }
  }
  __syncthreads();
  for (int i = tid; i < kChunk * kChunk; i += kPrepThreads)
    split_store(Ah + (i / kChunk) * kARow + i % kChunk, Al + (i / kChunk) * kARow + i % kChunk, sA[i]);
  if (tid < kChunk) floor_[tid] = (scalar && tid < len) ? gates[(size_t)(row + tid) * p.H + h].z : 1.f;
}

// ---------------------------------------------------------------------------------------
// chunk scan
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
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16x2(x - f.x, y - f.y);
}

constexpr int kScanStages = 4;
constexpr int kScanMaxWarps = 12;

struct ScanSmem {
  int tile, v_row, v_off, g_off, stage, obuf_off, obuf_row, bar_off, total;
  __host__ __device__ ScanSmem(int dkp, int dvp, int dv) {
    tile = tile_bytes(dkp);
    v_row = dvp + 8;
    v_off = (tile + 15) / 16 * 16;
    g_off = v_off + kChunk * v_row * 2;
    stage = (g_off + kChunk * dv * 2 + 127) / 128 * 128;
    obuf_off = kScanStages * stage;
    obuf_row = dvp + 4;
    bar_off = obuf_off + 2 * kChunk * obuf_row * 4;
    total = bar_off + kScanStages * 8;
  }
};

// warp w of the CTA owns value columns 16 w .. 16 w + 15 (rows of the fragment), all key channels (NK steps of 16)
template <int NK>
__global__ void __launch_bounds__(32 * kScanMaxWarps)
chunk_scan_kernel(RecParams p, const int* __restrict__ seq_chunk0, const int* __restrict__ slots,
                  const int* __restrict__ pos0, const int* __restrict__ chunk_row, const int* __restrict__ chunk_len,
                  const uint8_t* __restrict__ tiles, int* status) {
  constexpr int dkp = NK * 16;
  extern __shared__ __align__(128) uint8_t smem[];
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int dvp = (p.dv + norm + 15) / 16 * 16;
  const ScanSmem L(dkp, dvp, p.dv);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + L.bar_off);
  float* obuf = reinterpret_cast<float*>(smem + L.obuf_off);
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_warps = blockDim.x >> 5;
  const int c0 = seq_chunk0[s], n = seq_chunk0[s + 1] - c0, slot = slots[s];
  if (n <= 0 || slot < 0) return;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x);
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + p.out_off + (size_t)h * p.dv;

  if (tid == 0) {
    for (int i = 0; i < kScanStages; ++i) mbar_init(&full[i], 1);
    fence_barrier_init();
  }
  // value tiles: rows and columns that no copy writes stay finite; the normaliser's column is one
  for (int st = 0; st < kScanStages; ++st) {
    __nv_bfloat16* v = reinterpret_cast<__nv_bfloat16*>(smem + st * L.stage + L.v_off);
    for (int i = tid; i < kChunk * L.v_row; i += blockDim.x)
      v[i] = __float2bfloat16(norm && i % L.v_row == p.dv ? 1.f : 0.f);
  }
  fence_proxy_async_smem();
  __syncthreads();

  auto issue = [&](int c) {      // warp 0: copies of chunk c into its stage
    uint8_t* st = smem + (c % kScanStages) * L.stage;
    uint64_t* bar = &full[c % kScanStages];
    const int len = chunk_len[c0 + c];
    if (lane == 0) {
      mbar_arrive_expect_tx(bar, (uint32_t)(L.tile + 2 * len * p.dv * 2));
      bulk_load(st, tiles + ((size_t)(c0 + c) * p.H + h) * L.tile, (uint32_t)L.tile, bar);
    }
    __syncwarp();
    if (lane < len) {
      const __nv_bfloat16* xr = x + (size_t)(chunk_row[c0 + c] + lane) * p.row_stride + h * p.dv;
      bulk_load(st + L.v_off + lane * L.v_row * 2, xr + p.v_off, (uint32_t)p.dv * 2, bar);
      bulk_load(st + L.g_off + lane * p.dv * 2, xr + p.g_off, (uint32_t)p.dv * 2, bar);
    }
  };
  int issued = 0;
  if (warp == 0)
    for (; issued < n && issued < kScanStages - 1; ++issued) issue(issued);

  // state fragments: acc[j] holds key channels 8 j + 2 (lane % 4) + {0, 1} of value columns r and r + 8
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  const int r = warp * 16 + g;
  const int rows = p.dv + norm;
  float* gs = p.S + ((size_t)slot * p.H + h) * rows * p.dk;
  float acc[2 * NK][4];
  const bool fresh = pos0[s] == 0;
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = r + (i >> 1) * 8, d = 8 * j + q2 + (i & 1);
      acc[j][i] = (!fresh && rr < rows && d < p.dk) ? gs[(size_t)rr * p.dk + d] : 0.f;
    }

  const int rs = tile_row(dkp);
  // lane's row / column offsets inside a 16 x 16 tile for the two ldmatrix arrangements
  const int nrm_row = (lane & 7) + ((lane >> 4) << 3), nrm_col = ((lane >> 3) & 1) * 8;   // pairs along n, then k
  const int trn_row = (lane & 7) + (((lane >> 3) & 1) << 3), trn_col = (lane >> 4) * 8;   // k rows, then n columns
  const int va_row = (lane & 7) + ((lane >> 4) << 3), va_col = ((lane >> 3) & 1) * 8;     // s rows, value columns
  bool ok = true;
  int c = 0;
  for (; c < n; ++c) {
    ok = mbar_wait(&full[c % kScanStages], (c / kScanStages) & 1, status, kStatusTimeoutEpilogue);
    const uint8_t* st = smem + (c % kScanStages) * L.stage;
    float o0[2][4] = {}, o1[2][4] = {}, o2[2][4] = {};
    if (ok) {
      const uint32_t aq = smem_u32(st), al = aq + kChunk * rs * 2, akh = al + kChunk * rs * 2, akl = akh + kChunk * rs * 2;
      const uint32_t aA = akl + kChunk * rs * 2, aAl = aA + kChunk * kARow * 2;
      const float* D = reinterpret_cast<const float*>(st + 4 * kChunk * rs * 2 + 2 * kChunk * kARow * 2);
      uint32_t va[4];
      ldsm_x4_t(va, smem_u32(st + L.v_off) + (uint32_t)(va_row * L.v_row + warp * 16 + va_col) * 2);
#pragma unroll
      for (int kk = 0; kk < NK; ++kk) {
        uint32_t hi[4], lo[4], bh[4], bl[4];
        split_pair(acc[2 * kk][0], acc[2 * kk][1], hi[0], lo[0]);
        split_pair(acc[2 * kk][2], acc[2 * kk][3], hi[1], lo[1]);
        split_pair(acc[2 * kk + 1][0], acc[2 * kk + 1][1], hi[2], lo[2]);
        split_pair(acc[2 * kk + 1][2], acc[2 * kk + 1][3], hi[3], lo[3]);
        const uint32_t off = (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2;
        ldsm_x4(bh, aq + off);
        ldsm_x4(bl, al + off);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_16816(o0[nt], hi, bh[2 * nt], bh[2 * nt + 1]);
          mma_16816(o1[nt], hi, bl[2 * nt], bl[2 * nt + 1]);
          mma_16816(o2[nt], lo, bh[2 * nt], bh[2 * nt + 1]);
        }
      }
      {
        uint32_t bh[4], bl[4];
        const uint32_t off = (uint32_t)(nrm_row * kARow + nrm_col) * 2;
        ldsm_x4(bh, aA + off);
        ldsm_x4(bl, aAl + off);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_16816(o1[nt], va, bh[2 * nt], bh[2 * nt + 1]);
          mma_16816(o2[nt], va, bl[2 * nt], bl[2 * nt + 1]);
        }
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
    }
    float* ob = obuf + (c & 1) * kChunk * L.obuf_row;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        ob[(nt * 8 + q2 + (i & 1)) * L.obuf_row + r + (i >> 1) * 8] = o0[nt][i] + o1[nt][i] + o2[nt][i];
    if (!__syncthreads_and(ok)) {
      ok = false;
      break;
    }
    // the stage of chunk c - 1 is free: every warp has finished that chunk's output
    if (warp == 0 && issued < n) issue(issued++);
    const int len = chunk_len[c0 + c];
    const float* floor_ = reinterpret_cast<const float*>(st + 4 * kChunk * rs * 2 + 2 * kChunk * kARow * 2) + dkp;
    const __nv_bfloat16* gt = reinterpret_cast<const __nv_bfloat16*>(st + L.g_off);
    for (int t = warp; t < len; t += n_warps) {
      const float* orow = ob + t * L.obuf_row;
      float inv = 1.f;
      if (norm) inv = 1.f / (fmaxf(fabsf(orow[p.dv]), floor_[t]) + 1e-6f);
      float ss = 0.f;
      for (int i = lane; i < p.dv; i += 32) ss += (orow[i] * inv) * (orow[i] * inv);
      const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
      const float f = inv * rstd * p.out_scale;
      const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.norm_w) + (p.norm_per_head ? h * p.dv : 0);
      __nv_bfloat16* dst = out + (size_t)(chunk_row[c0 + c] + t) * p.out_stride;
      for (int i = lane * 2; i < p.dv; i += 64) {
        const float2 o = *reinterpret_cast<const float2*>(orow + i);
        const float2 wv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(w + i));
        const float2 gv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gt + t * p.dv + i));
        *reinterpret_cast<uint32_t*>(dst + i) = pack_bf16x2(o.x * f * wv.x * gate_value(gv.x, p.gate_act),
                                                            o.y * f * wv.y * gate_value(gv.y, p.gate_act));
      }
    }
  }
  if (!ok) {      // let the copies in flight land before shared memory is given back
    if (warp == 0)
      for (int k = c; k < issued; ++k) mbar_wait(&full[k % kScanStages], (k / kScanStages) & 1, nullptr, 0);
    return;
  }
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = r + (i >> 1) * 8, d = 8 * j + q2 + (i & 1);
      if (rr < rows && d < p.dk) gs[(size_t)rr * p.dk + d] = acc[j][i];
    }
}

template <int NK>
static int launch_scan(const RecParams& p, const int* seq_chunk0, const int* slots, const int* pos0, const int* chunk_row,
                       const int* chunk_len, const uint8_t* tiles, int n_seq, int* status, cudaStream_t stream) {
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int dvp = (p.dv + norm + 15) / 16 * 16;
  const ScanSmem L(NK * 16, dvp, p.dv);
  auto kernel = chunk_scan_kernel<NK>;
  static int configured = 0;
  if (configured < L.total) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total);
    if (e != cudaSuccess) return (int)e;
    configured = L.total;
  }
  kernel<<<dim3(p.H, n_seq), dvp / 16 * 32, L.total, stream>>>(p, seq_chunk0, slots, pos0, chunk_row, chunk_len, tiles,
                                                               status);
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

// Bytes of workspace of sb_recurrence_prefill for `n_chunks` chunks and `T` rows, or -1 when the sizes need the
// token-by-token kernel (dk <= 128, dv a multiple of 8, dv (+1) <= 192, 16-byte aligned rows).
extern "C" long long sb_recurrence_workspace(const void* params, int n_chunks, int T) {
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  const int norm = p.kind == kGateHead ? 1 : 0;
  const int dkp = (p.dk + 15) / 16 * 16, dvp = (p.dv + norm + 15) / 16 * 16;
  if (dkp > 128 || p.dv % 8 || dvp > 16 * kScanMaxWarps || p.row_stride % 8 || p.v_off % 8 || p.g_off % 8 ||
      p.out_stride % 2 || p.out_off % 2 || p.rank > 256 || ((uintptr_t)p.x & 15) || ((uintptr_t)p.out & 3))
    return -1;
  return (long long)n_chunks * p.H * tile_bytes(dkp) + (long long)T * p.H * 16;
}

// bf16 prefill of packed portions in 16-token chunks: chunk c covers rows chunk_row[c] .. + chunk_len[c], sequence s has
// chunks seq_chunk0[s] .. seq_chunk0[s + 1].
extern "C" int sb_recurrence_prefill(const void* params, const int* row0, const int* nrow, const int* slots,
                                     const int* pos0, int n_seq, const int* seq_chunk0, const int* chunk_row,
                                     const int* chunk_len, int n_chunks, int T, void* workspace, int* status,
                                     cudaStream_t stream) {
  if (n_seq == 0 || n_chunks == 0) return 0;
  if (n_seq > 65535 || ((uintptr_t)workspace & 15)) return -3;
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  if (sb_recurrence_workspace(params, n_chunks, T) < 0) return -2;
  const int dkp = (p.dk + 15) / 16 * 16;
  float4* gates = reinterpret_cast<float4*>(workspace);
  uint8_t* tiles = reinterpret_cast<uint8_t*>(workspace) + (size_t)T * p.H * 16;
  if (p.kind == kGateHead) {
    gate_scan_kernel<<<dim3(p.H, n_seq), kGsThreads, 0, stream>>>(p, row0, nrow, slots, pos0, gates);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
  }
  const size_t smem = (size_t)(3 * kChunk * (dkp + 1) + kChunk * kChunk + (p.kind == kGateChannel ? kChunk * p.rank : 0)) * 4;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  chunk_prepare_kernel<<<dim3(n_chunks, p.H), kPrepThreads, smem, stream>>>(p, chunk_row, chunk_len, gates, tiles, dkp);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  switch (dkp / 16) {
#define SB_SCAN(NK) \
  case NK: return launch_scan<NK>(p, seq_chunk0, slots, pos0, chunk_row, chunk_len, tiles, n_seq, status, stream);
    SB_SCAN(1) SB_SCAN(2) SB_SCAN(3) SB_SCAN(4) SB_SCAN(5) SB_SCAN(6) SB_SCAN(7) SB_SCAN(8)
#undef SB_SCAN
  }
  return -2;
}
