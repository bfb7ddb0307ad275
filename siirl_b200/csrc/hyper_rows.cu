// Hyper-connections: a decoder keeps S copies of its residual stream in 32-bit floats, h [rows, S, W].  One launch stands
// between two sublayers:
//
//   y   = sum of partial products + bias + sum_j w_j expert_row[slot_j] + w_id * input row      (result of the one before)
//   h_t = sum_s mix[s, t] h_s + out[t] * y                                                      (all from the old copies)
//   u   = sum_s in[s] h_s                                                                       (the one that follows)
//   row = layer_norm(u) * w + b                                                                 (in the activation format)
//
// The first launch takes every copy from the embedding table instead, the last one sums the copies (in = null).
// The routed part reads the experts' rows where the grouped products left them: no launch combines them beforehand.
#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"

namespace sb {

// mirrored by a ctypes structure in ops/rows.py
struct HyperParams {
  float* h;                 // [rows, S, W]
  int rows, S, W, vocab;
  const long long* ids;     // [rows]: the copies start as rows of `table`; null: they are in h
  const void* table;        // [vocab, W]
  const void* y;            // [slabs, rows, W] partial sums (fp32), one tensor in the activation format, or null
  long long slab;
  int slabs, y_f32;
  const void* bias;         // [W] or null
  const void* ys;           // expert rows [.., W] in the activation format, or null
  const int* pair_slot;     // [rows, top] row of ys (-1: none)
  const float* pair_w;      // [rows, top]
  const float* w_id;        // [rows] weight of the input row, or null
  const void* x_id;         // [rows, W] input rows
  int top;
  float eps;
  const void* w_mix;        // [S, S] from, to; null: nothing to add, the copies stay as they are
  const void* w_out;        // [S]
  const void* w_in;         // [S]; null: all ones
  const void* norm_w;       // [W]
  const void* norm_b;       // [W]
  void* out;                // [rows, W]
};
static_assert(sizeof(HyperParams) == 168, "HyperParams is mirrored from Python");

constexpr int kHyperThreads = 256;
constexpr int kHyperMax = 16;       // copies of the stream

__device__ __forceinline__ float hyper_row_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = red[0];
#pragma unroll
  for (int i = 1; i < kHyperThreads / 32; ++i) t += red[i];
  return t;
}

// CH register chunks of V elements per thread hold u (CH = 0: it is read back from the copies); SN copies (0: any number, the
// loops over them stay loops)
template <typename T, int V, int CH, int SN>
__global__ void __launch_bounds__(kHyperThreads) hyper_rows_kernel(const __grid_constant__ HyperParams p) {
  __shared__ float red[kHyperThreads / 32];
  __shared__ float s_mix[kHyperMax * kHyperMax], s_out[kHyperMax], s_in[kHyperMax];
  constexpr int SM = SN ? SN : kHyperMax, UN = SN ? SN : 1;
  const int S = SN ? SN : p.S, W = p.W, nv = W / V;
  if (threadIdx.x < S * S && p.w_mix) s_mix[threadIdx.x] = to_float(reinterpret_cast<const T*>(p.w_mix)[threadIdx.x]);
  if (threadIdx.x < S) {
    if (p.w_mix) s_out[threadIdx.x] = to_float(reinterpret_cast<const T*>(p.w_out)[threadIdx.x]);
    s_in[threadIdx.x] = p.w_in ? to_float(reinterpret_cast<const T*>(p.w_in)[threadIdx.x]) : 1.f;
  }
  __syncthreads();
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    float* hr = p.h + (size_t)row * S * W;
    T* orow = reinterpret_cast<T*>(p.out) + (size_t)row * W;
    long long id = 0;
    if (p.ids) {
      id = p.ids[row];
      id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    }
    const float w_id = p.w_id ? p.w_id[row] : 0.f;
    // the new copies at vector vi, stored; u of the sublayer that follows
    auto fetch = [&](int vi, float (&u)[V]) {
      const size_t c = (size_t)vi * V;
      float x[SM][V];
      if (p.ids) {
        load_vec<T, V>(reinterpret_cast<const T*>(p.table) + (size_t)id * W + c, x[0]);
#pragma unroll UN
        for (int s = 1; s < SM; ++s)
          if (s < S) {
#pragma unroll
            for (int i = 0; i < V; ++i) x[s][i] = x[0][i];
          }
      } else {
#pragma unroll UN
        for (int s = 0; s < SM; ++s)
          if (s < S) load_vec<float, V>(hr + (size_t)s * W + c, x[s]);
      }
      if (p.w_mix) {
        float y[V] = {};
        const size_t at = (size_t)row * W + c;
        if (p.y) {
          if (p.y_f32) {
            const float* yp = reinterpret_cast<const float*>(p.y) + at;
            load_vec<float, V>(yp, y);
            for (int k = 1; k < p.slabs; ++k) {
              float a[V];
              load_vec<float, V>(yp + k * p.slab, a);
#pragma unroll
              for (int i = 0; i < V; ++i) y[i] += a[i];
            }
          } else {
            load_vec<T, V>(reinterpret_cast<const T*>(p.y) + at, y);
          }
        }
        if (p.bias) {
          float b[V];
          load_vec<T, V>(reinterpret_cast<const T*>(p.bias) + c, b);
#pragma unroll
          for (int i = 0; i < V; ++i) y[i] += b[i];
        }
        if (p.ys) {
          for (int j = 0; j < p.top; ++j) {
            const int slot = p.pair_slot[(size_t)row * p.top + j];
            if (slot < 0) continue;
            const float w = p.pair_w[(size_t)row * p.top + j];
            float e[V];
            load_vec<T, V>(reinterpret_cast<const T*>(p.ys) + (size_t)slot * W + c, e);
#pragma unroll
            for (int i = 0; i < V; ++i) y[i] = fmaf(w, e[i], y[i]);
          }
        }
        if (p.w_id && w_id != 0.f) {
          float e[V];
          load_vec<T, V>(reinterpret_cast<const T*>(p.x_id) + at, e);
#pragma unroll
          for (int i = 0; i < V; ++i) y[i] = fmaf(w_id, e[i], y[i]);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) {
          float n[SM];
#pragma unroll UN
          for (int t = 0; t < SM; ++t) {
            if (t >= S) break;
            float a = s_out[t] * y[i];
#pragma unroll UN
            for (int s = 0; s < SM; ++s)
              if (s < S) a = fmaf(s_mix[s * S + t], x[s][i], a);
            n[t] = a;
          }
#pragma unroll UN
          for (int t = 0; t < SM; ++t)
            if (t < S) x[t][i] = n[t];
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = 0.f;
#pragma unroll UN
      for (int s = 0; s < SM; ++s) {
        if (s >= S) break;
        if (p.ids || p.w_mix) store_vec<float, V>(hr + (size_t)s * W + c, x[s]);
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] = fmaf(s_in[s], x[s][i], u[i]);
      }
    };
    float u[CH > 0 ? CH : 1][V];
    auto each = [&](auto&& fn) {
      if constexpr (CH > 0) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
          const int vi = threadIdx.x + c * kHyperThreads;
          if (vi < nv) fn(vi, u[c]);
        }
      } else {
        for (int vi = threadIdx.x; vi < nv; vi += kHyperThreads) {
#pragma unroll
          for (int i = 0; i < V; ++i) u[0][i] = 0.f;
          for (int s = 0; s < S; ++s) {      // written by this same thread above
            float x[V];
            load_vec<float, V>(hr + (size_t)s * W + (size_t)vi * V, x);
#pragma unroll
            for (int i = 0; i < V; ++i) u[0][i] = fmaf(s_in[s], x[i], u[0][i]);
          }
          fn(vi, u[0]);
        }
      }
    };
    float s = 0.f;
    if constexpr (CH > 0) {
#pragma unroll
      for (int c = 0; c < CH; ++c) {
        const int vi = threadIdx.x + c * kHyperThreads;
        if (vi < nv) {
          fetch(vi, u[c]);
#pragma unroll
          for (int i = 0; i < V; ++i) s += u[c][i];
        }
      }
    } else {
      for (int vi = threadIdx.x; vi < nv; vi += kHyperThreads) {
        fetch(vi, u[0]);
#pragma unroll
        for (int i = 0; i < V; ++i) s += u[0][i];
      }
    }
    const float mean = hyper_row_sum(s, red) / (float)W;
    float ss = 0.f;
    each([&](int, float (&v)[V]) {
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(v[i] - mean, v[i] - mean, ss);
    });
    const float f = 1.f / sqrtf(hyper_row_sum(ss, red) / (float)W + p.eps);
    each([&](int vi, float (&v)[V]) {
      float w[V], b[V], o[V];
      load_vec<T, V>(reinterpret_cast<const T*>(p.norm_w) + (size_t)vi * V, w);
      load_vec<T, V>(reinterpret_cast<const T*>(p.norm_b) + (size_t)vi * V, b);
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = fmaf((v[i] - mean) * f, w[i], b[i]);
      store_vec<T, V>(orow + (size_t)vi * V, o);
    });
  }
}

template <typename T, int V, int CH>
static int launch_hyper(const HyperParams& p, cudaStream_t s) {
  const int grid = p.rows < num_sms() * 8 ? p.rows : num_sms() * 8;
  switch (p.S) {
    case 1: hyper_rows_kernel<T, V, CH, 1><<<grid, kHyperThreads, 0, s>>>(p); break;
    case 2: hyper_rows_kernel<T, V, CH, 2><<<grid, kHyperThreads, 0, s>>>(p); break;
    case 3: hyper_rows_kernel<T, V, CH, 3><<<grid, kHyperThreads, 0, s>>>(p); break;
    case 4: hyper_rows_kernel<T, V, CH, 4><<<grid, kHyperThreads, 0, s>>>(p); break;
    default: hyper_rows_kernel<T, 1, 0, 0><<<grid, kHyperThreads, 0, s>>>(p); break;
  }
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_hyper_rows(const HyperParams& p, cudaStream_t s) {
  const int W = p.W;
  if constexpr (sizeof(T) == 2) {
    if (W % 8 == 0 && W <= 8 * kHyperThreads) return launch_hyper<T, 8, 1>(p, s);
    if (W % 8 == 0 && W <= 2 * 8 * kHyperThreads) return launch_hyper<T, 8, 2>(p, s);
  }
  if (W % 4) return launch_hyper<T, 1, 0>(p, s);
  if (W <= 4 * kHyperThreads) return launch_hyper<T, 4, 1>(p, s);
  if (W <= 4 * 4 * kHyperThreads) return launch_hyper<T, 4, 4>(p, s);
  return launch_hyper<T, 4, 0>(p, s);
}

}  // namespace sb

using namespace sb;

// params: host HyperParams; f32: activations and weights are fp32 (else bf16)
extern "C" int sb_hyper_rows(const void* params, int f32, cudaStream_t stream) {
  const HyperParams& p = *reinterpret_cast<const HyperParams*>(params);
  if (p.rows <= 0) return 0;
  if (p.S < 1 || p.S > kHyperMax || p.W < 1 || (p.ids && !p.table) || (p.w_mix && !p.w_out) || (p.w_id && !p.x_id) ||
      (p.ys && !(p.pair_slot && p.pair_w)))
    return -3;
  return f32 ? launch_hyper_rows<float>(p, stream) : launch_hyper_rows<__nv_bfloat16>(p, stream);
}
