// Generalized delta rule with a matrix state, for prefill and for decode (arguments and state layout of recurrence.cuh):
//
//   S_t = diag(w_t) S_(t-1) - b_t (u_t^T S_(t-1)) + k_t v_t^T          o_t = S_t^T r_t
//
// per sequence and head, state in 32-bit floats, with the unit key u = k / sqrt(|k|^2 + 1e-6), b = sigmoid(a + bias) * u, the
// decay w = exp(-e^(-1/2) sigmoid(W2 tanh(low-rank row) + bias)) per key channel; then an RMS norm of every head, a weight
// per channel and an output gate.  State: S [slots, heads, dv, dk], value-major; a portion whose first position is 0 starts from
// zero and does not read its slot.
//
// A chunk of 16 tokens.  With the decay G_t from the chunk's start through token t, r~ = G_t r_t, u~ = G_(t-1) u_t,
// k~ = k_t / G_t, b~ = b_t / G_t and p_t = u_t^T S_(t-1):
//
//   p_t = u~_t S_0 + sum_(s<t) (u~_t . k~_s) v_s - (u~_t . b~_s) p_s
//   o_t = r~_t S_0 + sum_(s<=t) (r~_t . k~_s) v_s - (r~_t . b~_s) p_s
//   S_16 = G (S_0 + sum_s k~_s v_s^T - b~_s p_s^T)
//
// The first line is a unit lower triangular system in p.  Solving it for the parts that multiply S_0 and v gives tiles that do
// not depend on the state, U = (I + ub)^-1 u~ and M = (I + ub)^-1 uk, and with them Q = r~ - rb U, A = rk - rb M,
// K = G (k~ - M^T b~), B = G b~:
//
//   o = Q S_0 + A v        p' = U S_0        S_16 = G S_0 + K^T v - B^T p'
//
// 1 / G_t is at most 2^14 inside a chunk (w > 0.54); the tiles are formed relative to the chunk's middle.
//
// Kernels:
//   delta_step_regs_kernel   one CTA per (sequence, head), the state in registers, token by token: decode, 32-bit prompts
//   delta_step_kernel        the same for any sizes, state in shared or global memory
//   delta_lowrank_kernel     prefill: tanh of the low-rank rows as two bf16 terms, once for all heads
//   delta_prepare_kernel     prefill: the tiles of a chunk, in parallel over chunks and heads.  (I + ub)^-1 itself by forward
//                            substitution in fp32, its products on the tensor cores
//   delta_scan_kernel        prefill: walks the chunks of a segment of a (sequence, head) with the state in registers as
//                            tensor-core fragments; tiles arrive through a ring of asynchronous copies.  Long prompts are cut
//                            into segments that run in parallel: a first pass makes each segment's state from zero and, as
//                            further value columns that start as the identity, the matrix its start state is multiplied by;
//                            delta_chain_kernel makes the start states, a second pass the outputs
// Tensor-core operands that stand for 32-bit quantities are split into two bf16 terms (16 mantissa bits), v is bf16 as projected;
// accumulation is fp32.
#include "recurrence.cuh"

namespace sb {

constexpr float kDecayRate = 0.6065306597126334f;      // e^(-1/2)

// decays, unit keys and removal rates of one token of head h, for all threads of a CTA of kStepThreads: sq (r), sk, su, sb, sd [dk].
// `se` holds rank values, `red` eight.  Ends with a barrier.
template <typename T>
__device__ __forceinline__ void delta_token(const RecParams& p, const T* xr, int h, float* sq, float* sk, float* su, float* sb_,
                                            float* sd, float* se, float* red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int r = tid; r < p.rank; r += kStepThreads) se[r] = tanhf(to_float(xr[p.e_off + r]));
  float ss = 0.f;
  for (int d = tid; d < p.dk; d += kStepThreads) {
    const float k = to_float(xr[p.k_off + h * p.dk + d]);
    sk[d] = k;
    sq[d] = to_float(xr[p.q_off + h * p.dk + d]);
    ss = fmaf(k, k, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < kStepThreads / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot + 1e-6f);
  const bool vec = sizeof(T) == 2 && p.rank % 8 == 0 && ((uintptr_t)p.w2 & 15) == 0;
  const int part = tid & 3;      // four lanes share a channel's product with the low-rank row
  for (int i = tid; i < (p.dk * 4 + 31) / 32 * 32; i += kStepThreads) {
    const int d = i >> 2;
    float z = 0.f;
    if (d < p.dk) {
      const T* w = reinterpret_cast<const T*>(p.w2) + (size_t)(h * p.dk + d) * p.rank;
      if constexpr (sizeof(T) == 2) {
        if (vec) {
          for (int r = part * 8; r < p.rank; r += 32) {
            float x[8];
            load_vec<T, 8>(w + r, x);
#pragma unroll
            for (int j = 0; j < 8; ++j) z = fmaf(x[j], se[r + j], z);
          }
        }
      }
      if (!vec)
        for (int r = part; r < p.rank; r += 4) z = fmaf(to_float(w[r]), se[r], z);
    }
    z += __shfl_xor_sync(0xffffffffu, z, 1);
    z += __shfl_xor_sync(0xffffffffu, z, 2);
    if (d < p.dk && part == 0) {
      z += to_float(reinterpret_cast<const T*>(p.b_e)[h * p.dk + d]);
      const float a = to_float(xr[p.f_off + h * p.dk + d]) + to_float(reinterpret_cast<const T*>(p.b_f)[h * p.dk + d]);
      sd[d] = expf(-kDecayRate / (1.f + expf(-z)));
      const float u = sk[d] * inv;
      su[d] = u;
      sb_[d] = u / (1.f + expf(-a));
    }
  }
  __syncthreads();
}

// norm, weight and gate of one token's head `so` [dv]; begins with a barrier (so is complete), red: eight values
template <typename T>
__device__ __forceinline__ void delta_finish(const RecParams& p, const T* xr, T* out, int h, const float* so, float* red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  __syncthreads();
  float ss = 0.f;
  for (int i = tid; i < p.dv; i += kStepThreads) ss = fmaf(so[i], so[i], ss);
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
    out[i] = from_float<T>(so[i] * rstd * w * g * p.out_scale);
  }
}

// rows of shared memory of the step kernels: five vectors of dk, so [dv], se [rank], two reductions
__host__ __device__ inline int delta_step_floats(int dk, int dv, int rank) {
  return 5 * ((dk + 3) & ~3) + ((dv + 3) & ~3) + ((rank + 3) & ~3) + 16;
}

// dk = dv <= 32 N, a multiple of four.  Eight lanes hold a state row (a value column's key channels), four rows per warp and pass.
// Everything a token needs is asked for at once, before the first barrier: a decoding step waits for memory twice, for its slot
// and for the rest.
template <typename T, int N>
__global__ void __launch_bounds__(kStepThreads, N <= 2 ? 4 : 2)
delta_step_regs_kernel(RecParams p, const int* __restrict__ row0, const int* __restrict__ nrow,
                       const int* __restrict__ slots, const int* __restrict__ pos0) {
  extern __shared__ __align__(16) float sm[];
  const int dkp = (p.dk + 3) & ~3;
  float *sq = sm, *sk = sq + dkp, *su = sk + dkp, *sb_ = su + dkp, *sd = sb_ + dkp, *so = sd + dkp;
  float *se = so + ((p.dv + 3) & ~3), *red = se + ((p.rank + 3) & ~3);
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
  const int r0 = row0 ? row0[s] : s, n = nrow ? nrow[s] : 1, slot = slots[s];
  T* out = reinterpret_cast<T*>(p.out) + p.out_off + (size_t)h * p.dv;
  if (slot < 0) {
    for (int t = 0; t < n; ++t)
      for (int i = tid; i < p.dv; i += kStepThreads) out[(size_t)(r0 + t) * p.out_stride + i] = from_float<T>(0.f);
    return;
  }
  if (n <= 0) return;
  const bool fresh = pos0[s] == 0;
  float* gs = p.S + ((size_t)slot * p.H + h) * p.dv * p.dk;
  const int warp = tid >> 5, lane = tid & 31, row = warp * 4 + (lane >> 3), d0 = (lane & 7) * 4;
  float st[N][N][4];      // [row row + 32 i][channels d0 + 32 c ..]
#pragma unroll
  for (int i = 0; i < N; ++i)
#pragma unroll
    for (int c = 0; c < N; ++c) {
#pragma unroll
      for (int j = 0; j < 4; ++j) st[i][c][j] = 0.f;
      if (!fresh && row + 32 * i < p.dv && d0 + 32 * c < p.dk)
        load_vec<float, 4>(gs + (size_t)(row + 32 * i) * p.dk + d0 + 32 * c, st[i][c]);
    }
  // four lanes share a channel's product with the low-rank row: channels tid / 4 and, for wide heads, + 64
  constexpr int CN = (N + 1) / 2;
  const int part = tid & 3;
  const bool vec = sizeof(T) == 2 && p.rank % 8 == 0 && ((uintptr_t)p.w2 & 15) == 0;
  float b_e[CN], b_f[CN];
  uint4 w_pre[CN][2];      // this lane's first sixteen weights
#pragma unroll
  for (int c = 0; c < CN; ++c) {
    const int d = (tid >> 2) + 64 * c;
    b_e[c] = b_f[c] = 0.f;
    w_pre[c][0] = w_pre[c][1] = make_uint4(0, 0, 0, 0);
    if (d >= p.dk) continue;
    b_e[c] = to_float(reinterpret_cast<const T*>(p.b_e)[h * p.dk + d]);
    b_f[c] = to_float(reinterpret_cast<const T*>(p.b_f)[h * p.dk + d]);
    if constexpr (sizeof(T) == 2) {
#pragma unroll
      for (int k = 0; k < 2; ++k)
        if (vec && part * 8 + 32 * k < p.rank)
          w_pre[c][k] = *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p.w2) + (size_t)(h * p.dk + d) * p.rank + part * 8 + 32 * k);
    }
  }
  const float nw = tid < p.dv ? to_float(reinterpret_cast<const T*>(p.norm_w)[p.norm_per_head ? h * p.dv + tid : tid]) : 0.f;
  for (int t = 0; t < n; ++t) {
    const T* xr = reinterpret_cast<const T*>(p.x) + (size_t)(r0 + t) * p.row_stride;
    const float k_in = tid < p.dk ? to_float(xr[p.k_off + h * p.dk + tid]) : 0.f;
    const float q_in = tid < p.dk ? to_float(xr[p.q_off + h * p.dk + tid]) : 0.f;
    const float g_in = tid < p.dv ? to_float(xr[p.g_off + h * p.dv + tid]) : 0.f;
    float a_in[CN], v[N], o[N], seen[N];
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      const int d = (tid >> 2) + 64 * c;
      a_in[c] = d < p.dk ? to_float(xr[p.f_off + h * p.dk + d]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      v[i] = row + 32 * i < p.dv ? to_float(xr[p.v_off + h * p.dv + row + 32 * i]) : 0.f;
      o[i] = seen[i] = 0.f;
    }
    for (int r = tid; r < p.rank; r += kStepThreads) se[r] = tanhf(to_float(xr[p.e_off + r]));
    if (tid < p.dk) {
      sk[tid] = k_in;
      sq[tid] = q_in;
    }
    float ss = warp_sum(k_in * k_in);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) tot += red[i];
    const float inv = 1.f / sqrtf(tot + 1e-6f);
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      const int d = (tid >> 2) + 64 * c;
      float z = 0.f;
      if (d < p.dk) {
        const T* w = reinterpret_cast<const T*>(p.w2) + (size_t)(h * p.dk + d) * p.rank;
        if constexpr (sizeof(T) == 2) {
          if (vec) {
            for (int r = part * 8, k = 0; r < p.rank; r += 32, ++k) {
              float x[8];
              if (k == 0) load_vec<T, 8>(reinterpret_cast<const T*>(&w_pre[c][0]), x);
              else if (k == 1) load_vec<T, 8>(reinterpret_cast<const T*>(&w_pre[c][1]), x);
              else load_vec<T, 8>(w + r, x);
              const float4 e0 = *reinterpret_cast<const float4*>(se + r), e1 = *reinterpret_cast<const float4*>(se + r + 4);
              z = fmaf(x[0], e0.x, fmaf(x[1], e0.y, fmaf(x[2], e0.z, fmaf(x[3], e0.w, z))));
              z = fmaf(x[4], e1.x, fmaf(x[5], e1.y, fmaf(x[6], e1.z, fmaf(x[7], e1.w, z))));
            }
          }
        }
        if (!vec)
          for (int r = part; r < p.rank; r += 4) z = fmaf(to_float(w[r]), se[r], z);
      }
      z += __shfl_xor_sync(0xffffffffu, z, 1);
      z += __shfl_xor_sync(0xffffffffu, z, 2);
      if (d < p.dk && part == 0) {
        sd[d] = expf(-kDecayRate / (1.f + expf(-(z + b_e[c]))));
        const float u = sk[d] * inv;
        su[d] = u;
        sb_[d] = u / (1.f + expf(-(a_in[c] + b_f[c])));
      }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < N; ++c) {
      if (d0 + 32 * c >= p.dk) break;
      float u[4];
      load_vec<float, 4>(su + d0 + 32 * c, u);
#pragma unroll
      for (int i = 0; i < N; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) seen[i] = fmaf(u[j], st[i][c][j], seen[i]);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      seen[i] += __shfl_xor_sync(0xffffffffu, seen[i], 4);
      seen[i] += __shfl_xor_sync(0xffffffffu, seen[i], 2);
      seen[i] += __shfl_xor_sync(0xffffffffu, seen[i], 1);
    }
#pragma unroll
    for (int c = 0; c < N; ++c) {
      if (d0 + 32 * c >= p.dk) break;
      float w[4], b[4], k[4], q[4];
      load_vec<float, 4>(sd + d0 + 32 * c, w);
      load_vec<float, 4>(sb_ + d0 + 32 * c, b);
      load_vec<float, 4>(sk + d0 + 32 * c, k);
      load_vec<float, 4>(sq + d0 + 32 * c, q);
#pragma unroll
      for (int i = 0; i < N; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float x = fmaf(st[i][c][j], w[j], fmaf(k[j], v[i], -b[j] * seen[i]));
          st[i][c][j] = x;
          o[i] = fmaf(x, q[j], o[i]);
        }
    }
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      o[i] += __shfl_xor_sync(0xffffffffu, o[i], 4);
      o[i] += __shfl_xor_sync(0xffffffffu, o[i], 2);
      o[i] += __shfl_xor_sync(0xffffffffu, o[i], 1);
      o[i] *= p.q_scale;
      if ((lane & 7) == 0 && row + 32 * i < p.dv) {
        so[row + 32 * i] = o[i];
        ss = fmaf(o[i], o[i], ss);
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[8 + warp] = ss;
    __syncthreads();
    tot = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) tot += red[8 + i];
    const float rstd = 1.f / sqrtf(tot / (float)p.dv + p.eps);
    if (tid < p.dv)
      out[(size_t)(r0 + t) * p.out_stride + tid] = from_float<T>(so[tid] * rstd * nw * gate_value(g_in, p.gate_act) * p.out_scale);
  }
#pragma unroll
  for (int i = 0; i < N; ++i)
#pragma unroll
    for (int c = 0; c < N; ++c)
      if (row + 32 * i < p.dv && d0 + 32 * c < p.dk)
        store_vec<float, 4>(gs + (size_t)(row + 32 * i) * p.dk + d0 + 32 * c, st[i][c]);
}

template <typename T>
__global__ void __launch_bounds__(kStepThreads)
delta_step_kernel(RecParams p, const int* __restrict__ row0, const int* __restrict__ nrow, const int* __restrict__ slots,
                  const int* __restrict__ pos0, int smem_state) {
  extern __shared__ __align__(16) float sm[];
  const int dkp = (p.dk + 3) & ~3;
  float *sq = sm, *sk = sq + dkp, *su = sk + dkp, *sb_ = su + dkp, *sd = sb_ + dkp, *so = sd + dkp;
  float *se = so + ((p.dv + 3) & ~3), *red = se + ((p.rank + 3) & ~3);
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
  const int r0 = row0 ? row0[s] : s, n = nrow ? nrow[s] : 1, slot = slots[s];
  T* out = reinterpret_cast<T*>(p.out) + p.out_off + (size_t)h * p.dv;
  if (slot < 0) {
    for (int t = 0; t < n; ++t)
      for (int i = tid; i < p.dv; i += kStepThreads) out[(size_t)(r0 + t) * p.out_stride + i] = from_float<T>(0.f);
    return;
  }
  if (n <= 0) return;
  const bool fresh = pos0[s] == 0;
  float* gs = p.S + ((size_t)slot * p.H + h) * p.dv * p.dk;
  float* st = smem_state ? red + 16 : gs;
  if (smem_state || fresh)
    for (int i = tid; i < p.dv * p.dk; i += kStepThreads) st[i] = fresh ? 0.f : gs[i];
  const int warp = tid >> 5, lane = tid & 31, grp = lane >> 3, l8 = lane & 7;
  for (int t = 0; t < n; ++t) {
    const T* xr = reinterpret_cast<const T*>(p.x) + (size_t)(r0 + t) * p.row_stride;
    delta_token<T>(p, xr, h, sq, sk, su, sb_, sd, se, red);
    for (int rb = warp * 4; rb < p.dv; rb += kStepThreads / 8) {
      const int r = rb + grp;
      float* sr = st + (size_t)(r < p.dv ? r : 0) * p.dk;
      float seen = 0.f, o = 0.f;
      if (r < p.dv)
        for (int d = l8; d < p.dk; d += 8) seen = fmaf(su[d], sr[d], seen);
      for (int w = 4; w; w >>= 1) seen += __shfl_xor_sync(0xffffffffu, seen, w);
      if (r < p.dv) {
        const float v = to_float(xr[p.v_off + h * p.dv + r]);
        for (int d = l8; d < p.dk; d += 8) {
          const float x = fmaf(sr[d], sd[d], fmaf(sk[d], v, -sb_[d] * seen));
          sr[d] = x;
          o = fmaf(x, sq[d], o);
        }
      }
      for (int w = 4; w; w >>= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
      if (l8 == 0 && r < p.dv) so[r] = o * p.q_scale;
    }
    delta_finish<T>(p, xr, out + (size_t)(r0 + t) * p.out_stride, h, so, red + 8);
  }
  if (smem_state) {
    __syncthreads();
    for (int i = tid; i < p.dv * p.dk; i += kStepThreads) gs[i] = st[i];
  }
}

// ---------------------------------------------------------------------------------------
// chunk tiles: Q, U, K, B [16][dkp + 8], each as hi and lo, then A hi, lo [16][24], then the chunk's decay [dkp] fp32
// ---------------------------------------------------------------------------------------
__host__ __device__ inline int delta_tile_bytes(int dkp) {
  return 8 * kChunk * tile_row(dkp) * 2 + 2 * kChunk * kARow * 2 + dkp * 4;
}

constexpr int kDeltaThreads = 128;

struct DeltaPrepSmem {      // byte offsets
  int cum, ub, small, e, inv, total;
  __host__ __device__ DeltaPrepSmem(int dkp, int rankp) {
    cum = delta_tile_bytes(dkp);                                     // [16][dkp + 1] running log2 decay
    ub = (cum + kChunk * (dkp + 1) * 4 + 15) / 16 * 16;              // [16][16] fp32
    small = ub + kChunk * kChunk * 4;                                // rk, rb, uk, inverse: [16][24], hi and lo
    e = small + 8 * kChunk * kARow * 2;                              // low-rank rows, hi and lo [16][rankp + 8]
    inv = e + 2 * kChunk * (rankp + 8) * 2;                          // [16][dkp / 8] squares of the keys
    total = inv + kChunk * (dkp / 8) * 4;
  }
};

// absolute error of a few 1e-7: it enters a sum that a sigmoid follows
__device__ __forceinline__ float delta_tanh(float x) { return 1.f - __fdividef(2.f, 1.f + __expf(2.f * x)); }
// log2 of the decay: -e^(-1/2) log2(e) sigmoid(z)
__device__ __forceinline__ float delta_log2_decay(float z) { return __fdividef(-kDecayRate * kLog2e, 1.f + __expf(-z)); }

// rows [T][2][rankp]: tanh of the low-rank rows as hi and lo, zeros past the rank
__global__ void delta_lowrank_kernel(RecParams p, long long total, int rankp, __nv_bfloat16* __restrict__ rows) {
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + p.e_off;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / rankp;
    const int r = (int)(i - t * rankp);
    const float e = r < p.rank ? delta_tanh(to_float(x[t * p.row_stride + r])) : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16(e);
    rows[t * 2 * rankp + r] = hi;
    rows[t * 2 * rankp + rankp + r] = __float2bfloat16(e - __bfloat162float(hi));
  }
}

// two neighbours from their two-term form
__device__ __forceinline__ float2 joined(uint32_t hi, uint32_t lo) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&lo));
  return make_float2(a.x + b.x, a.y + b.y);
}
__device__ __forceinline__ void stsm_x4_t(uint32_t addr, const uint32_t (&r)[4]) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]),
               "r"(r[3]) : "memory");
}
// Fragments of a 16 x 16 matrix: c[n][i] is the accumulator's form (row g + 8 (i / 2), column 8 n + 2 (lane % 4) + i % 2); as a
// left operand its pairs are (n, i / 2) = 00, 01, 10, 11.
struct Frag {
  float c[2][4];
};
__device__ __forceinline__ void frag_split(const Frag& f, float s0, float s1, uint32_t (&hi)[4], uint32_t (&lo)[4]) {      // rows g, g + 8 times s0, s1
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    split_pair(f.c[n][0] * s0, f.c[n][1] * s0, hi[2 * n], lo[2 * n]);
    split_pair(f.c[n][2] * s1, f.c[n][3] * s1, hi[2 * n + 1], lo[2 * n + 1]);
  }
}
__device__ __forceinline__ void frag_join(const uint32_t (&hi)[4], const uint32_t (&lo)[4], Frag& f) {
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float2 v = joined(hi[2 * n + e], lo[2 * n + e]);
      f.c[n][2 * e] = v.x;
      f.c[n][2 * e + 1] = v.y;
    }
}
// f += A B, both in two terms; b[2 n], b[2 n + 1]: columns 8 n ..
__device__ __forceinline__ void frag_mma(Frag& f, const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[4],
                                         const uint32_t (&bl)[4]) {
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    mma_16816(f.c[n], ah, bh[2 * n], bh[2 * n + 1]);
    mma_16816(f.c[n], ah, bl[2 * n], bl[2 * n + 1]);
    mma_16816(f.c[n], al, bh[2 * n], bh[2 * n + 1]);
  }
}

template <int NK>
__global__ void __launch_bounds__(kDeltaThreads)
delta_prepare_kernel(RecParams p, const int* __restrict__ chunk_row, const int* __restrict__ chunk_len,
                     const __nv_bfloat16* __restrict__ lowrank, int rankp, uint8_t* __restrict__ tiles) {
  using B16 = __nv_bfloat16;
  constexpr int dkp = NK * 16, rs = dkp + 8, ld = dkp + 1;
  const DeltaPrepSmem L(dkp, rankp);
  extern __shared__ __align__(16) uint8_t smem[];
  B16* t_q = reinterpret_cast<B16*>(smem);      // every tile: hi, then lo `part` elements later
  constexpr int part = kChunk * rs;
  B16 *t_u = t_q + 2 * part, *t_k = t_q + 4 * part, *t_b = t_q + 6 * part, *t_a = t_q + 8 * part;
  float* t_d = reinterpret_cast<float*>(t_a + 2 * kChunk * kARow);
  float* cum = reinterpret_cast<float*>(smem + L.cum);
  float* m_ub = reinterpret_cast<float*>(smem + L.ub);
  constexpr int mat = kChunk * kARow;           // small matrices: hi, then lo `mat` elements later
  B16 *m_rk = reinterpret_cast<B16*>(smem + L.small), *m_rb = m_rk + 2 * mat, *m_uk = m_rk + 4 * mat, *m_inv = m_rk + 6 * mat;
  B16* s_e = reinterpret_cast<B16*>(smem + L.e);
  const int e_part = kChunk * (rankp + 8);
  float* s_sq = reinterpret_cast<float*>(smem + L.inv);
  const int h = blockIdx.x, c = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row = chunk_row[c], len = chunk_len[c];
  const B16* x = reinterpret_cast<const B16*>(p.x) + (size_t)row * p.row_stride;
  const B16* w2 = reinterpret_cast<const B16*>(p.w2) + (size_t)h * p.dk * p.rank;
  const B16* w0 = reinterpret_cast<const B16*>(p.b_e) + h * p.dk;
  const B16* ab = reinterpret_cast<const B16*>(p.b_f) + h * p.dk;

  // a thread's vectors of eight channels of r, k, a: under way while the decays are made
  constexpr int per = dkp / 8, items = (kChunk * per + kDeltaThreads - 1) / kDeltaThreads;
  uint4 raw[items][3];
#pragma unroll
  for (int it = 0; it < items; ++it) {
    const int i = tid + it * kDeltaThreads, t = i / per, d = i % per * 8;
#pragma unroll
    for (int m = 0; m < 3; ++m) raw[it][m] = make_uint4(0, 0, 0, 0);
    if (t < len && d < p.dk) {
      const B16* xr = x + (size_t)t * p.row_stride + h * p.dk + d;
      raw[it][0] = *reinterpret_cast<const uint4*>(xr + p.k_off);
      raw[it][1] = *reinterpret_cast<const uint4*>(xr + p.q_off);
      raw[it][2] = *reinterpret_cast<const uint4*>(xr + p.f_off);
    }
  }
  {      // low-rank rows; eight threads per token
    const int t = tid >> 3;
    const B16* src = lowrank + (size_t)(row + t) * 2 * rankp;
    for (int e = (tid & 7) * 8; e < 2 * rankp; e += 64) {
      B16* dst = s_e + (e < rankp ? t * (rankp + 8) + e : e_part + t * (rankp + 8) + e - rankp);
      if (t < len) copy16(dst, src + e);
      else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
    copy_commit();
    copy_wait<0>();
  }
  __syncthreads();
  // log2 decays: rows t = g, g + 8, channels 8 j + 2 (lane % 4) + {0, 1} of a warp's column groups
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  const int nrm_row = (lane & 7) + ((lane >> 4) << 3), nrm_col = ((lane >> 3) & 1) * 8;
  const int trn_row = (lane & 7) + (((lane >> 3) & 1) << 3), trn_col = (lane >> 4) * 8;
  const bool whole = p.rank == rankp && ((uintptr_t)w2 & 3) == 0;
  const uint32_t a_e = smem_u32(s_e) + (uint32_t)(trn_row * (rankp + 8) + trn_col) * 2;
  for (int j = warp; j < dkp / 8; j += kDeltaThreads / 32) {
    float z[4] = {}, z2[4] = {};
    const int ch = 8 * j + g;      // the channel whose weights this lane brings
    const B16* w = w2 + (size_t)(ch < p.dk ? ch : 0) * p.rank + q2;
#pragma unroll 4
    for (int k0 = 0; k0 < rankp; k0 += 16, w += 16) {
      uint32_t a[4], b[2] = {0, 0};
      if (whole) {
        b[0] = *reinterpret_cast<const uint32_t*>(w);
        b[1] = *reinterpret_cast<const uint32_t*>(w + 8);
      } else {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = k0 + q2 + 8 * half;
          if (r < p.rank) b[half] = pack_bf16x2(to_float(w[8 * half]), r + 1 < p.rank ? to_float(w[8 * half + 1]) : 0.f);
        }
      }
      ldsm_x4(a, a_e + k0 * 2);
      mma_16816(z, a, b[0], b[1]);
      ldsm_x4(a, a_e + (e_part + k0) * 2);
      mma_16816(z2, a, b[0], b[1]);
    }
    const int d = 8 * j + q2;      // d + 1 lies below dk with d: dk is a multiple of eight
    const float b0 = d < p.dk ? to_float(w0[d]) : 0.f, b1 = d < p.dk ? to_float(w0[d + 1]) : 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = g + (i >> 1) * 8;
      cum[t * ld + d + (i & 1)] = t < len && d < p.dk ? delta_log2_decay(z[i] + z2[i] + (i & 1 ? b1 : b0)) : 0.f;
    }
  }
#pragma unroll
  for (int it = 0; it < items; ++it) {
    const int i = tid + it * kDeltaThreads;
    float k[8], ss = 0.f;
    load_vec<B16, 8>(reinterpret_cast<const B16*>(&raw[it][0]), k);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(k[j], k[j], ss);
    if (i < kChunk * per) s_sq[i] = ss;
  }
  __syncthreads();
  for (int d = tid; d < dkp; d += kDeltaThreads) {
    float acc = 0.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      acc += cum[t * ld + d];
      cum[t * ld + d] = acc;
    }
    t_d[d] = ex2(acc);
  }
  __syncthreads();
  // r~, u~, k~, b~ relative to the decay through token 7
#pragma unroll
  for (int it = 0; it < items; ++it) {
    const int i = tid + it * kDeltaThreads, t = i / per, d = i % per * 8;
    if (kChunk * per % kDeltaThreads && i >= kChunk * per) break;
    float r[8], k[8], a[8], bias[8] = {}, ss = 0.f;
    load_vec<B16, 8>(reinterpret_cast<const B16*>(&raw[it][0]), k);
    load_vec<B16, 8>(reinterpret_cast<const B16*>(&raw[it][1]), r);
    load_vec<B16, 8>(reinterpret_cast<const B16*>(&raw[it][2]), a);
    if (d < p.dk) load_vec<B16, 8>(ab + d, bias);
#pragma unroll
    for (int j = 0; j < per; ++j) ss += s_sq[t * per + j];
    const float inv = rsqrtf(ss + 1e-6f);
    uint32_t out[8][4];
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      float v[4][2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float mid = cum[7 * ld + d + j + e], now = cum[t * ld + d + j + e];
        const float before = t ? cum[(t - 1) * ld + d + j + e] : 0.f;
        const float up = ex2(mid - now), u = k[j + e] * inv;
        v[0][e] = r[j + e] * p.q_scale * ex2(now - mid);
        v[1][e] = u * ex2(before - mid);
        v[2][e] = k[j + e] * up;
        v[3][e] = u * up * __fdividef(1.f, 1.f + __expf(-(a[j + e] + bias[j + e])));
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) split_pair(v[m][0], v[m][1], out[2 * m][j / 2], out[2 * m + 1][j / 2]);
    }
#pragma unroll
    for (int m = 0; m < 8; ++m)
      *reinterpret_cast<uint4*>(t_q + m * part + t * rs + d) = make_uint4(out[m][0], out[m][1], out[m][2], out[m][3]);
  }
  __syncthreads();
  // the four 16 x 16 products: warp w takes r~ or u~ (w / 2) with k~ or b~ (w % 2)
  {
    const B16 *X = warp >> 1 ? t_u : t_q, *Y = warp & 1 ? t_b : t_k;
    Frag pr = {}, pr2 = {};
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      uint32_t xh[4], xl[4], yh[4], yl[4];
      const uint32_t ax = smem_u32(X) + (uint32_t)(trn_row * rs + kk * 16 + trn_col) * 2;
      const uint32_t ay = smem_u32(Y) + (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2;
      ldsm_x4(xh, ax);
      ldsm_x4(xl, ax + part * 2);
      ldsm_x4(yh, ay);
      ldsm_x4(yl, ay + part * 2);
      frag_mma(kk & 1 ? pr2 : pr, xh, xl, yh, yl);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        const int t = g + (i >> 1) * 8, s = n * 8 + q2, last = t - (warp >> 1);      // s <= t, or s < t for u~
        const float v0 = s <= last ? pr.c[n][i] + pr2.c[n][i] : 0.f, v1 = s + 1 <= last ? pr.c[n][i + 1] + pr2.c[n][i + 1] : 0.f;
        if (warp == 3) {
          *reinterpret_cast<float2*>(m_ub + t * kChunk + s) = make_float2(v0, v1);
        } else {
          B16* m = m_rk + warp * 2 * mat + t * kARow + s;
          split_pair(v0, v1, *reinterpret_cast<uint32_t*>(m), *reinterpret_cast<uint32_t*>(m + mat));
        }
      }
  }
  __syncthreads();
  // (I + ub)^-1, one column per lane
  if (warp == 3) {
    if (lane < kChunk) {
      float sol[kChunk];
#pragma unroll
      for (int t = 0; t < kChunk; ++t) {
        float v[2] = {t == lane ? 1.f : 0.f, 0.f};
#pragma unroll
        for (int s4 = 0; s4 < t; s4 += 4) {
          const float4 l4 = *reinterpret_cast<const float4*>(m_ub + t * kChunk + s4);
          const float l[4] = {l4.x, l4.y, l4.z, l4.w};
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (s4 + e < t) v[e & 1] = fmaf(-l[e], sol[s4 + e], v[e & 1]);
        }
        sol[t] = v[0] + v[1];
        const B16 hi = __float2bfloat16(sol[t]);
        m_inv[t * kARow + lane] = hi;
        m_inv[mat + t * kARow + lane] = __float2bfloat16(sol[t] - __bfloat162float(hi));
      }
    }
  }
  __syncthreads();
  // Everything transposed, channels as rows: U^T = u~^T inv^T, Q^T = r~^T - U^T rb^T, M^T = uk^T inv^T, K^T = k~^T - b~^T M; A^T = rk^T - M^T rb^T
  {
    const uint32_t o_nrm = (uint32_t)(nrm_row * kARow + nrm_col) * 2, o_trn = (uint32_t)(nrm_row * kARow + nrm_col) * 2;
    uint32_t ih[4], il[4], rbh[4], rbl[4], mh[4], ml[4];
    ldsm_x4(ih, smem_u32(m_inv) + o_nrm);
    ldsm_x4(il, smem_u32(m_inv + mat) + o_nrm);
    ldsm_x4(rbh, smem_u32(m_rb) + o_nrm);
    ldsm_x4(rbl, smem_u32(m_rb + mat) + o_nrm);
    {
      uint32_t uh[4], ul[4];
      ldsm_x4_t(uh, smem_u32(m_uk) + o_trn);
      ldsm_x4_t(ul, smem_u32(m_uk + mat) + o_trn);
      Frag m = {};
      frag_mma(m, uh, ul, ih, il);
      frag_split(m, -1.f, -1.f, mh, ml);      // -M^T as a left operand; as a right operand of M's columns its pairs 1 and 2 change places
    }
    if (warp == 3) {
      uint32_t kh[4], kl[4], ah[4], al[4];
      ldsm_x4_t(kh, smem_u32(m_rk) + o_trn);
      ldsm_x4_t(kl, smem_u32(m_rk + mat) + o_trn);
      Frag a;
      frag_join(kh, kl, a);
      frag_mma(a, mh, ml, rbh, rbl);
      frag_split(a, 1.f, 1.f, ah, al);
      stsm_x4_t(smem_u32(t_a) + o_trn, ah);
      stsm_x4_t(smem_u32(t_a + mat) + o_trn, al);
    }
    const uint32_t bmh[4] = {mh[0], mh[2], mh[1], mh[3]}, bml[4] = {ml[0], ml[2], ml[1], ml[3]};
#pragma unroll 1
    for (int kk = warp; kk < NK; kk += kDeltaThreads / 32) {
      const uint32_t off = (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2;
      auto tile = [&](B16* t, int lo) { return smem_u32(t) + lo * part * 2 + off; };
      const int d0 = kk * 16 + g, d1 = d0 + 8;
      const float mid0 = cum[7 * ld + d0], mid1 = cum[7 * ld + d1];
      const float f0 = ex2(mid0), f1 = ex2(mid1);                                               // from the middle to the start
      const float e0 = ex2(cum[15 * ld + d0] - mid0), e1 = ex2(cum[15 * ld + d1] - mid1);       // and to the end
      uint32_t hi[4], lo[4], xh[4], xl[4];
      ldsm_x4_t(hi, tile(t_u, 0));
      ldsm_x4_t(lo, tile(t_u, 1));
      Frag u = {}, r;
      frag_mma(u, hi, lo, ih, il);
      frag_split(u, f0, f1, xh, xl);
      stsm_x4_t(tile(t_u, 0), xh);
      stsm_x4_t(tile(t_u, 1), xl);
      frag_split(u, -1.f, -1.f, xh, xl);
      ldsm_x4_t(hi, tile(t_q, 0));
      ldsm_x4_t(lo, tile(t_q, 1));
      frag_join(hi, lo, r);
      frag_mma(r, xh, xl, rbh, rbl);
      frag_split(r, f0, f1, xh, xl);
      stsm_x4_t(tile(t_q, 0), xh);
      stsm_x4_t(tile(t_q, 1), xl);
      ldsm_x4_t(hi, tile(t_k, 0));
      ldsm_x4_t(lo, tile(t_k, 1));
      frag_join(hi, lo, r);
      ldsm_x4_t(hi, tile(t_b, 0));
      ldsm_x4_t(lo, tile(t_b, 1));
      frag_mma(r, hi, lo, bmh, bml);
      frag_split(r, e0, e1, xh, xl);
      stsm_x4_t(tile(t_k, 0), xh);
      stsm_x4_t(tile(t_k, 1), xl);
      frag_join(hi, lo, r);
      frag_split(r, e0, e1, xh, xl);
      stsm_x4_t(tile(t_b, 0), xh);
      stsm_x4_t(tile(t_b, 1), xl);
    }
  }
  __syncthreads();
  uint8_t* tile = tiles + ((size_t)c * p.H + h) * delta_tile_bytes(dkp);
  for (int i = tid * 16; i < delta_tile_bytes(dkp); i += kDeltaThreads * 16)
    *reinterpret_cast<uint4*>(tile + i) = *reinterpret_cast<const uint4*>(smem + i);
}

// ---------------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------------
constexpr int kDeltaStages = 3;
constexpr int kDeltaGates = kDeltaStages + 1;      // gates are used one chunk later than the rest

struct DeltaScanSmem {
  int tile, v_row, v_off, stage, obuf_off, obuf_row, obuf, norm_off, gate_off, gate, total;
  __host__ __device__ DeltaScanSmem(int dkp, int dvp) {
    tile = delta_tile_bytes(dkp);
    v_row = dvp + 8;
    v_off = tile;
    stage = (v_off + kChunk * v_row * 2 + 127) / 128 * 128;
    obuf_off = kDeltaStages * stage;
    obuf_row = dvp + 4;
    obuf = kChunk * obuf_row;
    norm_off = obuf_off + 2 * obuf * 4;
    gate_off = norm_off + dvp * 4;
    gate = kChunk * dvp * 2;
    total = gate_off + kDeltaGates * gate;
  }
};

// Warp w owns value columns 16 w .. 16 w + 15 and all key channels.  OUT: iteration c multiplies chunk c and finishes (norm,
// gate, store) chunk c - 1: one block barrier per chunk.  Without OUT (the first pass over a segment that another one follows)
// the warps behind those of the values carry the identity along: what they end with is the segment's matrix.
template <int NK, bool OUT>
__global__ void __launch_bounds__(NK * (OUT ? 32 : 64), NK > 4 ? 1 : 2)
delta_scan_kernel(RecParams p, Segments sg, const int* __restrict__ slots, const int* __restrict__ pos0,
                  const uint8_t* __restrict__ tiles) {
  constexpr int dkp = NK * 16, rs = dkp + 8, KD = (dkp + 63) / 64, part = kChunk * rs * 2;      // part: bytes of one tile half
  extern __shared__ __align__(128) uint8_t smem[];
  const int dvp = (p.dv + 15) / 16 * 16;
  const DeltaScanSmem L(dkp, dvp);
  float* obuf = reinterpret_cast<float*>(smem + L.obuf_off);
  float* nw = reinterpret_cast<float*>(smem + L.norm_off);
  const int h = blockIdx.x, g_id = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_warps = blockDim.x >> 5;
  const int s = sg.seq[g_id], slot = slots[s], flags = sg.flags[g_id];
  const int tokens = sg.tokens[g_id], n = (tokens + kChunk - 1) / kChunk, row0 = sg.row[g_id];
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)row0 * p.row_stride;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)row0 * p.out_stride + p.out_off + (size_t)h * p.dv;
  if (slot < 0) {
    if (OUT)
      for (int i = tid; i < tokens * p.dv; i += blockDim.x)
        out[(size_t)(i / p.dv) * p.out_stride + i % p.dv] = __float2bfloat16(0.f);
    return;
  }
  if (n <= 0 || (!OUT && (flags & 2))) return;
  const uint8_t* my_tiles = tiles + ((size_t)sg.chunk0[g_id] * p.H + h) * L.tile;
  const size_t tile_step = (size_t)p.H * L.tile;
  for (int st = 0; st < kDeltaStages; ++st) {      // value columns past dv: no copy writes them
    __nv_bfloat16* v = reinterpret_cast<__nv_bfloat16*>(smem + st * L.stage + L.v_off);
    const int extra = L.v_row - p.dv;
    for (int i = tid; i < kChunk * extra; i += blockDim.x) v[i / extra * L.v_row + p.dv + i % extra] = __float2bfloat16(0.f);
  }
  // the place of a thread's first vector of the value rows does not change from chunk to chunk
  const int v_vecs = p.dv / 8, v_t = tid / v_vecs, v_e = (tid - v_t * v_vecs) * 8;
  const __nv_bfloat16 *v_src = x + p.v_off + h * p.dv, *g_src = x + p.g_off + h * p.dv;
  auto copy_v = [&](uint8_t* st, int c, int len, int t, int e) {
    uint8_t* dst = st + L.v_off + (t * L.v_row + e) * 2;
    if (t < len) copy16(dst, v_src + (size_t)(c * kChunk + t) * p.row_stride + e);
    else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
  };
  auto issue = [&](int c) {      // copies of chunk c into its stage (an empty group past the end)
    if (c < n) {
      uint8_t* st = smem + (c % kDeltaStages) * L.stage;
      const int len = min(kChunk, tokens - c * kChunk);
      const uint8_t* src = my_tiles + (size_t)c * tile_step;
      for (int i = tid * 16 + (OUT ? 0 : 2 * part); i < L.tile; i += blockDim.x * 16) copy16(st + i, src + i);
      if (v_t < kChunk) copy_v(st, c, len, v_t, v_e);
      for (int i = tid + blockDim.x; i < kChunk * v_vecs; i += blockDim.x) copy_v(st, c, len, i / v_vecs, i % v_vecs * 8);
      if constexpr (OUT) {
        uint8_t* gates = smem + L.gate_off + (c % kDeltaGates) * L.gate;
        for (int i = tid; i < len * v_vecs; i += blockDim.x) {
          const int t = i < (int)blockDim.x ? v_t : i / v_vecs, e = i < (int)blockDim.x ? v_e : i % v_vecs * 8;
          copy16(gates + (t * dvp + e) * 2, g_src + (size_t)(c * kChunk + t) * p.row_stride + e);
        }
      }
    }
    copy_commit();
  };
#pragma unroll
  for (int i = 0; i < kDeltaStages - 1; ++i) issue(i);

  // state fragments: acc[j] holds key channels 8 j + 2 (lane % 4) + {0, 1} of value columns r and r + 8
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  const bool carry = !OUT && warp >= dvp / 16;      // columns of the identity
  const int r = (carry ? warp - dvp / 16 : warp) * 16 + g;
  float* slot_S = p.S + ((size_t)slot * p.H + h) * p.dv * p.dk;
  float* seg_S = sg.S + ((size_t)g_id * p.H + h) * p.dv * p.dk;
  const bool single = (flags & 3) == 3;
  const float* from = single ? slot_S : seg_S;
  const bool zero = !OUT || (single && pos0[s] == 0);
  float acc[2 * NK][4];
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = r + (i >> 1) * 8, d = 8 * j + q2 + (i & 1);
      acc[j][i] = (!zero && rr < p.dv && d < p.dk) ? from[(size_t)rr * p.dk + d] : (carry && rr == d ? 1.f : 0.f);
    }
  if (OUT)
    for (int i = tid; i < p.dv; i += blockDim.x)
      nw[i] = to_float(reinterpret_cast<const __nv_bfloat16*>(p.norm_w)[(p.norm_per_head ? h * p.dv : 0) + i]);
  const float inv_dv = 1.f / (float)p.dv;
  const int nrm_row = (lane & 7) + ((lane >> 4) << 3), nrm_col = ((lane >> 3) & 1) * 8;   // rows 0-7: columns 0-7, 8-15
  const int trn_row = (lane & 7) + (((lane >> 3) & 1) << 3), trn_col = (lane >> 4) * 8;   // columns 0-7: rows 0-7, 8-15

  for (int c = 0; c <= n; ++c) {
    if (c < n) copy_wait<kDeltaStages - 2>();
    else if (!OUT) break;
    __syncthreads();            // chunk c has landed, chunk c - 1 is multiplied, chunk c - 2 is out
    issue(c + kDeltaStages - 1);
    if (c < n) {
      const uint8_t* st = smem + (c % kDeltaStages) * L.stage;
      const uint32_t a_q = smem_u32(st), a_u = a_q + 2 * part, a_k = a_q + 4 * part, a_b = a_q + 6 * part, a_a = a_q + 8 * part;
      const float* D = reinterpret_cast<const float*>(st + 8 * part + 2 * kChunk * kARow * 2);
      float* ob = obuf + (c & 1) * L.obuf;
      uint32_t va[4];             // v^T: value columns x tokens
      if (!carry) ldsm_x4_t(va, smem_u32(st + L.v_off) + (uint32_t)(nrm_row * L.v_row + warp * 16 + nrm_col) * 2);
      float p0[2][4] = {}, p1[2][4] = {}, p2[2][4] = {}, o0[2][4] = {}, o1[2][4] = {}, o2[2][4] = {};
#pragma unroll
      for (int kk = 0; kk < NK; ++kk) {
        uint32_t hi[4], lo[4], uh[4], ul[4];
        const uint32_t off = (uint32_t)(nrm_row * rs + kk * 16 + nrm_col) * 2;
        ldsm_x4(uh, a_u + off);
        ldsm_x4(ul, a_u + part + off);
        split_pair(acc[2 * kk][0], acc[2 * kk][1], hi[0], lo[0]);
        split_pair(acc[2 * kk][2], acc[2 * kk][3], hi[1], lo[1]);
        split_pair(acc[2 * kk + 1][0], acc[2 * kk + 1][1], hi[2], lo[2]);
        split_pair(acc[2 * kk + 1][2], acc[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_16816(p0[nt], hi, uh[2 * nt], uh[2 * nt + 1]);
          mma_16816(p1[nt], hi, ul[2 * nt], ul[2 * nt + 1]);
          mma_16816(p2[nt], lo, uh[2 * nt], uh[2 * nt + 1]);
        }
        if constexpr (OUT) {
          uint32_t qh[4], ql[4];
          ldsm_x4(qh, a_q + off);
          ldsm_x4(ql, a_q + part + off);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            mma_16816(o0[nt], hi, qh[2 * nt], qh[2 * nt + 1]);
            mma_16816(o1[nt], hi, ql[2 * nt], ql[2 * nt + 1]);
            mma_16816(o2[nt], lo, qh[2 * nt], qh[2 * nt + 1]);
          }
        }
      }
      // -p'^T as the left operand of the state update: the accumulator's places are those of a 16 x 16 operand
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          split_pair(-(p0[nt][2 * e] + p1[nt][2 * e] + p2[nt][2 * e]),
                     -(p0[nt][2 * e + 1] + p1[nt][2 * e + 1] + p2[nt][2 * e + 1]), ph[2 * nt + e], pl[2 * nt + e]);
#pragma unroll
      for (int kk = 0; kk < NK; ++kk) {
        uint32_t kh[4], kl[4], bh[4], bl[4];
        const uint32_t off = (uint32_t)(trn_row * rs + kk * 16 + trn_col) * 2;
        ldsm_x4_t(bh, a_b + off);
        ldsm_x4_t(bl, a_b + part + off);
        if (!carry) {
          ldsm_x4_t(kh, a_k + off);
          ldsm_x4_t(kl, a_k + part + off);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = 2 * kk + e;
          const float2 dd = *reinterpret_cast<const float2*>(D + 8 * j + q2);
          acc[j][0] *= dd.x;
          acc[j][1] *= dd.y;
          acc[j][2] *= dd.x;
          acc[j][3] *= dd.y;
          if (!carry) {
            mma_16816(acc[j], va, kh[2 * e], kh[2 * e + 1]);
            mma_16816(acc[j], va, kl[2 * e], kl[2 * e + 1]);
          }
          mma_16816(acc[j], ph, bh[2 * e], bh[2 * e + 1]);
          mma_16816(acc[j], ph, bl[2 * e], bl[2 * e + 1]);
          mma_16816(acc[j], pl, bh[2 * e], bh[2 * e + 1]);
        }
      }
      if constexpr (OUT) {
        uint32_t ah[4], al[4];
        const uint32_t off = (uint32_t)(nrm_row * kARow + nrm_col) * 2;
        ldsm_x4(ah, a_a + off);
        ldsm_x4(al, a_a + kChunk * kARow * 2 + off);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_16816(o1[nt], va, ah[2 * nt], ah[2 * nt + 1]);
          mma_16816(o2[nt], va, al[2 * nt], al[2 * nt + 1]);
#pragma unroll
          for (int i = 0; i < 4; ++i)
            ob[(nt * 8 + q2 + (i & 1)) * L.obuf_row + r + (i >> 1) * 8] = o0[nt][i] + o1[nt][i] + o2[nt][i];
        }
      }
    }
    if constexpr (OUT) {
      if (c == 0) continue;
      const float* ob = obuf + ((c - 1) & 1) * L.obuf;
      const int t0 = (c - 1) * kChunk, len = min(kChunk, tokens - t0);
      const __nv_bfloat16* gates = reinterpret_cast<const __nv_bfloat16*>(smem + L.gate_off + ((c - 1) % kDeltaGates) * L.gate);
      // each half warp finishes one token at a time: four values per lane and 64 columns
      for (int tb = warp * 2; tb < len; tb += n_warps * 2) {
        const int t = tb + (lane >> 4);      // below 16; rows past `len` are computed and not stored
        const float* orow = ob + t * L.obuf_row;
        float4 o[KD];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < KD; ++k) {
          const int i = (lane & 15) * 4 + k * 64;
          o[k] = i < p.dv ? *reinterpret_cast<const float4*>(orow + i) : make_float4(0.f, 0.f, 0.f, 0.f);
          ss += o[k].x * o[k].x + o[k].y * o[k].y + o[k].z * o[k].z + o[k].w * o[k].w;
        }
#pragma unroll
        for (int w = 8; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
        const float f = p.out_scale * rsqrtf(ss * inv_dv + p.eps);
        if (t >= len) continue;
        __nv_bfloat16* dst = out + (size_t)(t0 + t) * p.out_stride;
#pragma unroll
        for (int k = 0; k < KD; ++k) {
          const int i = (lane & 15) * 4 + k * 64;
          if (i >= p.dv) continue;
          const float4 w = *reinterpret_cast<const float4*>(nw + i);
          const uint2 graw = *reinterpret_cast<const uint2*>(gates + t * dvp + i);
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
  copy_wait<0>();
  if (OUT && !(flags & 2)) return;
  float* to = OUT ? slot_S : (carry ? sg.decay + ((size_t)g_id * p.H + h) * p.dk * p.dk : seg_S);
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = r + (i >> 1) * 8, d = 8 * j + q2 + (i & 1);
      if (rr < p.dv && d < p.dk) to[(size_t)rr * p.dk + d] = acc[j][i];
    }
}

// Start states of the segments of sequences that have several, in place of the states from zero: S <- S F + local, one segment
// after the other; the next matrix is copied while one is used.  A block has sixteen rows (value columns), a thread four of them
// and the channels d, d + 64, ..
constexpr int kChainRows = 16, kChainThreads = 256;
__host__ __device__ inline int chain_smem(int dk) { return (2 * dk * dk + 2 * kChainRows * dk) * 4; }

__global__ void __launch_bounds__(kChainThreads) delta_chain_kernel(RecParams p, Segments sg, const int* __restrict__ slots,
                                                                    const int* __restrict__ pos0) {
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x, d0 = tid & 63, grp = tid >> 6;
  const int slot = slots[s], g0 = sg.seq_seg0[s], g1 = sg.seq_seg0[s + 1], dk = p.dk;
  if (slot < 0 || g1 - g0 < 2) return;
  const int mat = dk * dk, v0 = blockIdx.x * kChainRows;
  float* state = sm + 2 * mat;      // [2][16][dk]
  auto copy = [&](int g) {          // the last segment's matrix is not needed
    if (g + 1 < g1) {
      const float* F = sg.decay + ((size_t)g * p.H + h) * mat;
      for (int i = tid * 4; i < mat; i += kChainThreads * 4) copy16(sm + ((g - g0) & 1) * mat + i, F + i);
    }
    copy_commit();
  };
  copy(g0);
  for (int i = tid; i < kChainRows * dk; i += kChainThreads) {
    const int v = v0 + i / dk;
    state[i] = pos0[s] == 0 || v >= p.dv ? 0.f : p.S[((size_t)slot * p.H + h) * p.dv * dk + (size_t)v0 * dk + i];
  }
  for (int g = g0; g < g1; ++g) {
    copy_wait<0>();
    __syncthreads();                // this matrix and this state are there, the other buffers have been read
    if (g + 1 < g1) copy(g + 1);
    const float* F = sm + ((g - g0) & 1) * mat;
    const float* now = state + (((g - g0) & 1) * kChainRows + grp * 4) * dk;
    float* next = state + ((((g - g0) & 1) ^ 1) * kChainRows + grp * 4) * dk;
    float* local = sg.S + ((size_t)g * p.H + h) * p.dv * dk + (size_t)(v0 + grp * 4) * dk;
    const int rows = min(4, p.dv - v0 - grp * 4);
    for (int d = d0; d < dk; d += 64) {
      float acc[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        acc[k] = g + 1 < g1 && k < rows ? local[k * dk + d] : 0.f;
        if (k < rows) local[k * dk + d] = now[k * dk + d];
      }
      if (g + 1 < g1) {
#pragma unroll 4
        for (int j = 0; j < dk; j += 4) {
          float4 n[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) n[k] = *reinterpret_cast<const float4*>(now + k * dk + j);
          const float f[4] = {F[j * dk + d], F[(j + 1) * dk + d], F[(j + 2) * dk + d], F[(j + 3) * dk + d]};
#pragma unroll
          for (int k = 0; k < 4; ++k) acc[k] = fmaf(n[k].x, f[0], fmaf(n[k].y, f[1], fmaf(n[k].z, f[2], fmaf(n[k].w, f[3], acc[k]))));
        }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) next[k * dk + d] = acc[k];
    }
  }
}

template <typename K>
static int delta_configure(K kernel, int smem, int& configured) {
  if (smem <= 48 * 1024 || smem <= configured) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return (int)e;
  configured = smem;
  return 0;
}

template <int NK>
static int launch_delta(const RecParams& p, const Segments& sg, int n_seg, const int* slots, const int* pos0, int n_seq,
                        const int* chunk_row, const int* chunk_len, int n_chunks, int T, __nv_bfloat16* lowrank, uint8_t* tiles,
                        cudaStream_t stream) {
  static int prep_smem = 0, scan_smem = 0, first_smem = 0;
  const int rankp = (p.rank + 15) / 16 * 16, psm = DeltaPrepSmem(NK * 16, rankp).total;
  const int dvp = (p.dv + 15) / 16 * 16, ssm = DeltaScanSmem(NK * 16, dvp).total;
  int r = delta_configure(delta_prepare_kernel<NK>, psm, prep_smem);
  if (r || (r = delta_configure(delta_scan_kernel<NK, true>, ssm, scan_smem)) ||
      (r = delta_configure(delta_scan_kernel<NK, false>, ssm, first_smem)))
    return r;
  cudaError_t e;
  const long long low = (long long)T * rankp;
  const long long blocks = (low + 255) / 256, most = (long long)num_sms() * 8;
  delta_lowrank_kernel<<<(int)(blocks < most ? blocks : most), 256, 0, stream>>>(p, low, rankp, lowrank);
  if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  // heads before chunks: the tiles of one chunk are neighbours in memory.  The grid's second dimension ends at 65535.
  for (int c = 0; c < n_chunks; c += 65535) {
    const int m = n_chunks - c < 65535 ? n_chunks - c : 65535;
    delta_prepare_kernel<NK><<<dim3(p.H, m), kDeltaThreads, psm, stream>>>(
        p, chunk_row + c, chunk_len + c, lowrank, rankp, tiles + (size_t)c * p.H * delta_tile_bytes(NK * 16));
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  }
  if (n_seg > n_seq) {
    delta_scan_kernel<NK, false><<<dim3(p.H, n_seg), dvp * 2 + NK * 32, ssm, stream>>>(p, sg, slots, pos0, tiles);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    static int chain_configured = 0;
    if ((r = delta_configure(delta_chain_kernel, chain_smem(p.dk), chain_configured))) return r;
    delta_chain_kernel<<<dim3((p.dv + kChainRows - 1) / kChainRows, p.H, n_seq), kChainThreads, chain_smem(p.dk), stream>>>(
        p, sg, slots, pos0);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
  }
  delta_scan_kernel<NK, true><<<dim3(p.H, n_seg), dvp * 2, ssm, stream>>>(p, sg, slots, pos0, tiles);
  return (int)cudaGetLastError();
}

}  // namespace sb

using namespace sb;

// Arguments of sb_recurrence_step: one token per sequence (row0 / nrow null) or a packed portion each, any sizes.
extern "C" int sb_delta_step(const void* params, const int* row0, const int* nrow, const int* slots, const int* pos0, int n_seq,
                             int f32, cudaStream_t stream) {
  if (n_seq == 0) return 0;
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  if (n_seq > 65535 || p.kind != kGateDelta || p.dk != p.dv || p.rank < 1 || !p.w2 || !p.b_e || !p.b_f) return -3;
  const size_t base = (size_t)delta_step_floats(p.dk, p.dv, p.rank) * 4;
  if (base > 100 * 1024) return -3;
  const dim3 grid(p.H, n_seq);
  if (p.dk % 4 == 0 && p.dk <= 128 && base <= 48 * 1024) {
    const int n = (p.dk + 31) / 32;
    auto run = [&](auto kernel) -> int {
      kernel<<<grid, kStepThreads, base, stream>>>(p, row0, nrow, slots, pos0);
      return (int)cudaGetLastError();
    };
    if (f32)
      return n == 1 ? run(delta_step_regs_kernel<float, 1>) : n == 2 ? run(delta_step_regs_kernel<float, 2>)
           : n == 3 ? run(delta_step_regs_kernel<float, 3>) : run(delta_step_regs_kernel<float, 4>);
    using H = __nv_bfloat16;
    return n == 1 ? run(delta_step_regs_kernel<H, 1>) : n == 2 ? run(delta_step_regs_kernel<H, 2>)
         : n == 3 ? run(delta_step_regs_kernel<H, 3>) : run(delta_step_regs_kernel<H, 4>);
  }
  const size_t state = (size_t)p.dv * p.dk * 4;
  const int in_smem = nrow != nullptr && base + state <= 200 * 1024;
  const size_t smem = base + (in_smem ? state : 0);
  auto run = [&](auto kernel) -> int {
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return (int)e;
    }
    kernel<<<grid, kStepThreads, smem, stream>>>(p, row0, nrow, slots, pos0, in_smem);
    return (int)cudaGetLastError();
  };
  return f32 ? run(delta_step_kernel<float>) : run(delta_step_kernel<__nv_bfloat16>);
}

// (segment, head) blocks of the scan that run at a time on the whole GPU
extern "C" int sb_delta_resident(const void* params) {
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  return num_sms() * (pad_dk(p.dk) > 64 ? 1 : 2);
}

// Bytes of workspace of sb_delta_prefill for `n_chunks` chunks, `n_seg` segments and `T` rows, or -1 when the sizes need sb_delta_step
// (head width a multiple of eight up to 128, 16-byte aligned rows).
extern "C" long long sb_delta_workspace(const void* params, int n_chunks, int n_seg, int T) {
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  if (p.kind != kGateDelta || p.dk != p.dv || p.dk % 8 || p.dk > 128 || p.row_stride % 8 || p.q_off % 8 || p.k_off % 8 ||
      p.v_off % 8 || p.f_off % 8 || p.g_off % 8 || p.out_stride % 4 || p.out_off % 4 || p.rank < 1 || p.rank > 512 ||
      ((uintptr_t)p.x & 15) || ((uintptr_t)p.out & 7) || ((uintptr_t)p.b_f & 15))
    return -1;
  return (long long)n_chunks * p.H * delta_tile_bytes(pad_dk(p.dk)) + (long long)n_seg * p.H * p.dk * p.dk * 8 +
         (long long)T * ((p.rank + 15) / 16 * 16) * 4;
}

// bf16 prefill of packed portions in 16-token chunks: chunk c covers rows chunk_row[c] .. + chunk_len[c].  Segments as in
// sb_recurrence_prefill: five int arrays of n_seg entries in `segs` (sequence, first chunk, first row, tokens, flags: 1 first, 2
// last), then n_seq + 1 entries with each sequence's first segment.
extern "C" int sb_delta_prefill(const void* params, const int* slots, const int* pos0, int n_seq, const int* chunk_row,
                                const int* chunk_len, int n_chunks, const int* segs, int n_seg, int T, void* workspace,
                                cudaStream_t stream) {
  if (n_seq == 0 || n_chunks == 0) return 0;
  if (n_seq > 65535 || n_seg > 65535 || ((uintptr_t)workspace & 15)) return -3;
  const RecParams& p = *reinterpret_cast<const RecParams*>(params);
  if (sb_delta_workspace(params, n_chunks, n_seg, T) < 0) return -2;
  uint8_t* tiles = reinterpret_cast<uint8_t*>(workspace);
  Segments sg;
  sg.seq = segs; sg.chunk0 = segs + n_seg; sg.row = segs + 2 * n_seg; sg.tokens = segs + 3 * n_seg;
  sg.flags = segs + 4 * n_seg; sg.seq_seg0 = segs + 5 * n_seg;
  sg.S = reinterpret_cast<float*>(tiles + (size_t)n_chunks * p.H * delta_tile_bytes(pad_dk(p.dk)));
  sg.decay = sg.S + (size_t)n_seg * p.H * p.dv * p.dk;
  __nv_bfloat16* lowrank = reinterpret_cast<__nv_bfloat16*>(sg.decay + (size_t)n_seg * p.H * p.dk * p.dk);
  switch (pad_dk(p.dk) / 16) {
#define SB_DELTA(NK) \
  case NK:           \
    return launch_delta<NK>(p, sg, n_seg, slots, pos0, n_seq, chunk_row, chunk_len, n_chunks, T, lowrank, tiles, stream);
    SB_DELTA(1) SB_DELTA(2) SB_DELTA(3) SB_DELTA(4) SB_DELTA(6) SB_DELTA(8)
#undef SB_DELTA
  }
  return -2;
}
