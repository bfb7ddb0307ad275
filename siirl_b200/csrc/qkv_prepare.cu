// What stands between the fused projection of an attention branch and its scores, one launch: sum of the projection's
// partial products, biases, RMS norms of queries and keys, rotation, append of keys and values to the paged cache
// (layout in win_params.h), queries in the activation format for the attention kernels, per-head output gates.  The
// branch's table of biases by distance is expanded from its buckets by blocks of its own.
//
//   norm 0  none
//   norm 1  a whole projection (all heads at once) over its root mean square times a weight vector, before the rotation
//   norm 2  every head over its root mean square, no weight, after the rotation
//
// Rotation: pairs (i, i + half) of the first 2 * half dimensions of a head turn by position * f_i.  f_i comes as two
// floats (hi + lo) and the angle keeps its remainder, so the error does not grow with the position.
//
// One block per row; a row's projections stay in shared memory as 32-bit floats between the sums and the stores.
#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"

namespace sb {

// mirrored by a ctypes structure in ops/window_attention.py
struct PrepareParams {
  const void* x;            // [slabs, T, row_stride] partial sums (fp32), or one tensor in the activation format
  long long slab, row_stride;
  int slabs, x_f32;
  const void* bias;         // [row_stride] columns like x, or null
  int q_off, k_off, v_off, g_off;   // g_off < 0: no gate
  int T, Hq, Hkv, dk, dv, norm;
  const void* q_norm;       // [Hq * dk] (norm 1)
  const void* k_norm;       // [Hkv * dk]
  float eps;
  int half;                 // rotated pairs per head
  const float* freq;        // [half, 2]
  const int* seq_ids;       // [T] cache slot of every row (-1: none)
  const int* positions;
  const int* block_table;   // [slots, max_blocks]
  void* cache;
  long long num_blocks, block_elems;
  int max_blocks, rel_n;
  void* q_out;              // [T, q_stride]
  long long q_stride;
  float* gate_out;          // [T, Hq] sigmoids, or null
  const void* rel;          // [buckets, Hq] distance table of the checkpoint, or null
  const int* bucket;        // [rel_n] its row for every distance
  float* rel_out;           // [Hq, rel_n]
};
static_assert(sizeof(PrepareParams) == 216, "PrepareParams is mirrored from Python");

constexpr int kPrepBlk = 64;        // tokens per cache block
constexpr int kPrepThreads = 128;

template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) qkv_prepare_kernel(const __grid_constant__ PrepareParams p) {
  extern __shared__ float sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if ((int)blockIdx.x >= p.T) {      // distance table
    const int n = p.Hq * p.rel_n, step = (gridDim.x - p.T) * kPrepThreads;
    for (int i = (blockIdx.x - p.T) * kPrepThreads + tid; i < n; i += step) {
      const int h = i / p.rel_n, d = i - h * p.rel_n;
      p.rel_out[i] = to_float(reinterpret_cast<const T*>(p.rel)[(size_t)p.bucket[d] * p.Hq + h]);
    }
    return;
  }
  const int t = blockIdx.x;
  const int nq = p.Hq * p.dk, nk = p.Hkv * p.dk, nv = p.Hkv * p.dv;
  float* s_x = sm;                    // [nq + nk]
  float* s_cos = s_x + nq + nk;       // [half]
  float* s_sin = s_cos + p.half;
  __shared__ float red[2][kPrepThreads / 32];
  const int slot = p.seq_ids[t], pos = p.positions[t];
  T* crow = nullptr;                  // this row's place in its cache block (head 0, keys)
  if (slot >= 0 && pos >= 0 && pos / kPrepBlk < p.max_blocks) {
    const int blk = p.block_table[(size_t)slot * p.max_blocks + pos / kPrepBlk];
    if (blk >= 0 && blk < p.num_blocks) crow = reinterpret_cast<T*>(p.cache) + (size_t)blk * p.block_elems;
  }
  const int place = pos % kPrepBlk;

  // V columns of the row from `col` on, summed over the partial products, with the bias
  auto fetch = [&](int col, float (&v)[V]) {
    const size_t at = (size_t)t * p.row_stride + col;
    if (p.x_f32) {
      const float* x = reinterpret_cast<const float*>(p.x) + at;
      load_vec<float, V>(x, v);
      for (int s = 1; s < p.slabs; ++s) {
        float y[V];
        load_vec<float, V>(x + s * p.slab, y);
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] += y[i];
      }
    } else {
      load_vec<T, V>(reinterpret_cast<const T*>(p.x) + at, v);
    }
    if (p.bias) {
      float b[V];
      load_vec<T, V>(reinterpret_cast<const T*>(p.bias) + col, b);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += b[i];
    }
  };
  float ssq = 0.f, ssk = 0.f;
  for (int e = tid * V; e < nq + nk; e += kPrepThreads * V) {
    float v[V];
    fetch(e < nq ? p.q_off + e : p.k_off + e - nq, v);
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      ss = fmaf(v[i], v[i], ss);
      s_x[e + i] = v[i];
    }
    if (e < nq) ssq += ss;
    else ssk += ss;
  }
  for (int e = tid * V; e < nv; e += kPrepThreads * V) {
    float v[V];
    fetch(p.v_off + e, v);
    const int head = e / p.dv;
    if (crow)
      store_vec<T, V>(crow + (size_t)p.Hkv * kPrepBlk * p.dk + ((size_t)head * kPrepBlk + place) * p.dv + (e - head * p.dv), v);
  }
  if (p.g_off >= 0) {
    for (int h = tid; h < p.Hq; h += kPrepThreads) {
      const size_t at = (size_t)t * p.row_stride + p.g_off + h;
      float z = 0.f;
      if (p.x_f32) {
        for (int s = 0; s < p.slabs; ++s) z += reinterpret_cast<const float*>(p.x)[s * p.slab + at];
      } else {
        z = to_float(reinterpret_cast<const T*>(p.x)[at]);
      }
      p.gate_out[(size_t)t * p.Hq + h] = 1.f / (1.f + expf(-z));
    }
  }
  for (int i = tid; i < p.half; i += kPrepThreads) {
    const float n = (float)pos, a = n * p.freq[2 * i], lo = fmaf(n, p.freq[2 * i], -a) + n * p.freq[2 * i + 1];
    float s, c;
    sincosf(a, &s, &c);
    s_cos[i] = fmaf(-s, lo, c);
    s_sin[i] = fmaf(c, lo, s);
  }
  float fq = 1.f, fk = 1.f;
  if (p.norm == 1) {
    ssq = warp_sum(ssq);
    ssk = warp_sum(ssk);
    if (lane == 0) {
      red[0][warp] = ssq;
      red[1][warp] = ssk;
    }
  }
  __syncthreads();
  if (p.norm == 1) {
    ssq = red[0][0] + red[0][1] + red[0][2] + red[0][3];
    ssk = red[1][0] + red[1][1] + red[1][2] + red[1][3];
    fq = 1.f / sqrtf(ssq / (float)nq + p.eps);
    fk = 1.f / sqrtf(ssk / (float)nk + p.eps);
  }

  constexpr int V2 = V == 1 ? 1 : 2;      // elements a lane turns and stores at once
  for (int h = warp; h < p.Hq + p.Hkv; h += kPrepThreads / 32) {
    const bool is_q = h < p.Hq;
    const int kh = h - p.Hq;
    const float* x = s_x + h * p.dk;
    float f = is_q ? fq : fk;
    if (p.norm == 2) {
      float ss = 0.f;
      for (int d = lane; d < p.dk; d += 32) ss = fmaf(x[d], x[d], ss);
      f = 1.f / sqrtf(warp_sum(ss) / (float)p.dk + p.eps);
    }
    const T* w = p.norm == 1 ? (is_q ? reinterpret_cast<const T*>(p.q_norm) + h * p.dk
                                     : reinterpret_cast<const T*>(p.k_norm) + kh * p.dk)
                             : nullptr;
    T* dst = is_q ? reinterpret_cast<T*>(p.q_out) + (size_t)t * p.q_stride + (size_t)h * p.dk
                  : (crow ? crow + ((size_t)kh * kPrepBlk + place) * p.dk : nullptr);
    if (!dst) continue;
    for (int d0 = lane * V2; d0 < p.dk; d0 += 32 * V2) {
      float o[V2];
#pragma unroll
      for (int i = 0; i < V2; ++i) {
        const int d = d0 + i;
        float a = x[d] * f;
        if (w) a *= to_float(w[d]);
        if (d < 2 * p.half) {
          const bool first = d < p.half;
          const int e = first ? d + p.half : d - p.half, r = first ? d : e;
          float b = x[e] * f;
          if (w) b *= to_float(w[e]);
          a = first ? fmaf(a, s_cos[r], -b * s_sin[r]) : fmaf(a, s_cos[r], b * s_sin[r]);
        }
        o[i] = a;
      }
      if constexpr (V2 == 1) {
        dst[d0] = from_float<T>(o[0]);
      } else if constexpr (sizeof(T) == 2) {
        *reinterpret_cast<uint32_t*>(dst + d0) = pack_bf16x2(o[0], o[1]);
      } else {
        *reinterpret_cast<float2*>(dst + d0) = make_float2(o[0], o[1]);
      }
    }
  }
}

template <typename T, int V>
static int launch_prepare(const PrepareParams& p, cudaStream_t s) {
  const size_t smem = ((size_t)(p.Hq + p.Hkv) * p.dk + 2 * (size_t)p.half) * 4;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (smem > 200 * 1024) return -3;
    cudaError_t e = cudaFuncSetAttribute(qkv_prepare_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  int extra = 0;
  if (p.rel) {
    extra = (p.Hq * p.rel_n + 4 * kPrepThreads - 1) / (4 * kPrepThreads);
    if (extra > num_sms()) extra = num_sms();
  }
  qkv_prepare_kernel<T, V><<<p.T + extra, kPrepThreads, smem, s>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace sb

using namespace sb;

// params: host PrepareParams; f32: activations, weights and cache are fp32 (else bf16)
extern "C" int sb_qkv_prepare(const void* params, int f32, cudaStream_t stream) {
  const PrepareParams& p = *reinterpret_cast<const PrepareParams*>(params);
  if (p.T <= 0) return 0;
  if (p.Hkv < 1 || p.Hq % p.Hkv || p.dk < 1 || p.dv < 1 || 2 * p.half > p.dk || p.slabs < 1 || (p.slabs > 1 && !p.x_f32) ||
      (p.norm == 1 && !(p.q_norm && p.k_norm)) || (p.half && !p.freq) || (p.g_off >= 0 && !p.gate_out) ||
      (p.rel && !(p.bucket && p.rel_out)))
    return -3;
  const int V = f32 ? 4 : 8;
  const bool vec = p.dk % V == 0 && p.dv % V == 0 && p.row_stride % V == 0 && p.slab % V == 0 && p.q_off % V == 0 &&
                   p.k_off % V == 0 && p.v_off % V == 0 && p.q_stride % V == 0 && p.block_elems % V == 0;
  if (f32) return vec ? launch_prepare<float, 4>(p, stream) : launch_prepare<float, 1>(p, stream);
  return vec ? launch_prepare<__nv_bfloat16, 8>(p, stream) : launch_prepare<__nv_bfloat16, 1>(p, stream);
}
