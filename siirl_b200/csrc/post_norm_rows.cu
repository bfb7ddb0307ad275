// Decoders with a norm before and behind every sublayer: what stands between two sublayers, one launch.  The residual stream h
// [rows, W] is kept in 32-bit floats:
//
//   y   = sum of partial products + bias + sum_j w_j expert_row[slot_j]          (result of the sublayer before)
//   h  += y / rms(y) * post
//   row = h / rms(h) * w     in the activation format (w = null: h itself, rounded)
//
// The first launch of a pass takes h from the embedding table, times a scale.  The routed part reads the experts' rows where the
// grouped products left them.
#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"

namespace sb {

// mirrored by a ctypes structure in ops/rows.py
struct PostNormParams {
  float* h;                 // [rows, W]
  int rows, W, vocab, top;
  const long long* ids;     // [rows]: h starts as rows of `table`; null: y is added
  const void* table;        // [vocab, W]
  float scale, eps;
  const void* y;            // [slabs, rows, W] partial sums (fp32), one tensor in the activation format, or null
  long long slab;
  int slabs, y_f32;
  const void* bias;         // [W] or null
  const void* ys;           // expert rows [.., W] in the activation format, or null
  const int* pair_slot;     // [rows, top] row of ys (-1: none)
  const float* pair_w;      // [rows, top]
  const void* post;         // [W] weight of y's norm
  const void* norm_w;       // [W] weight of the norm that follows, or null
  void* out;                // [rows, W]
};
static_assert(sizeof(PostNormParams) == 128, "PostNormParams is mirrored from Python");

constexpr int kPostThreads = 256;

__device__ __forceinline__ float post_row_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = red[0];
#pragma unroll
  for (int i = 1; i < kPostThreads / 32; ++i) t += red[i];
  return t;
}

// CH register chunks of V elements per thread hold y and then h (CH = 0: y is summed up again, h is read back)
template <typename T, int V, int CH>
__global__ void __launch_bounds__(kPostThreads) post_norm_rows_kernel(const __grid_constant__ PostNormParams p) {
  __shared__ float red[2][2][kPostThreads / 32];      // [row parity][sum]: one barrier per sum
  const int W = p.W, nv = W / V;
  int par = 0;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x, par ^= 1) {
    float* hr = p.h + (size_t)row * W;
    T* orow = reinterpret_cast<T*>(p.out) + (size_t)row * W;
    auto result = [&](int vi, float (&y)[V]) {
      const size_t c = (size_t)vi * V, at = (size_t)row * W + c;
#pragma unroll
      for (int i = 0; i < V; ++i) y[i] = 0.f;
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
    };
    constexpr int R = CH > 0 ? CH : 1;
    float x[R][V], hv[R][V];
    auto each = [&](auto&& fn) {      // fn(vector, register chunk)
      if constexpr (CH > 0) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
          const int vi = threadIdx.x + c * kPostThreads;
          if (vi < nv) fn(vi, c);
        }
      } else {
        for (int vi = threadIdx.x; vi < nv; vi += kPostThreads) fn(vi, 0);
      }
    };
    float ss = 0.f;
    if (p.ids) {
      long long id = p.ids[row];
      id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
      each([&](int vi, int c) {
        load_vec<T, V>(reinterpret_cast<const T*>(p.table) + (size_t)id * W + (size_t)vi * V, x[c]);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          x[c][i] *= p.scale;
          ss = fmaf(x[c][i], x[c][i], ss);
        }
        store_vec<float, V>(hr + (size_t)vi * V, x[c]);
      });
    } else {
      float sy = 0.f;
      if constexpr (CH > 0) each([&](int vi, int c) { load_vec<float, V>(hr + (size_t)vi * V, hv[c]); });
      each([&](int vi, int c) {
        result(vi, x[c]);
#pragma unroll
        for (int i = 0; i < V; ++i) sy = fmaf(x[c][i], x[c][i], sy);
      });
      const float f = 1.f / sqrtf(post_row_sum(sy, red[par][0]) / (float)W + p.eps);
      each([&](int vi, int c) {
        if constexpr (CH == 0) {
          load_vec<float, V>(hr + (size_t)vi * V, hv[c]);
          result(vi, x[c]);
        }
        float w[V];
        load_vec<T, V>(reinterpret_cast<const T*>(p.post) + (size_t)vi * V, w);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          x[c][i] = fmaf(x[c][i] * f, w[i], hv[c][i]);
          ss = fmaf(x[c][i], x[c][i], ss);
        }
        store_vec<float, V>(hr + (size_t)vi * V, x[c]);
      });
    }
    float f = 1.f;
    if (p.norm_w) f = 1.f / sqrtf(post_row_sum(ss, red[par][1]) / (float)W + p.eps);
    each([&](int vi, int c) {
      if constexpr (CH == 0) load_vec<float, V>(hr + (size_t)vi * V, x[c]);      // written by this same thread above
      if (p.norm_w) {
        float w[V];
        load_vec<T, V>(reinterpret_cast<const T*>(p.norm_w) + (size_t)vi * V, w);
#pragma unroll
        for (int i = 0; i < V; ++i) x[c][i] *= f * w[i];
      }
      store_vec<T, V>(orow + (size_t)vi * V, x[c]);
    });
  }
}

template <typename T, int V, int CH>
static int launch_post_norm(const PostNormParams& p, cudaStream_t s) {
  const int grid = p.rows < num_sms() * 8 ? p.rows : num_sms() * 8;
  post_norm_rows_kernel<T, V, CH><<<grid, kPostThreads, 0, s>>>(p);
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_post_norm_rows(const PostNormParams& p, cudaStream_t s) {
  const int W = p.W;
  if constexpr (sizeof(T) == 2) {
    if (W % 8 == 0 && W > 4 * kPostThreads && W <= 8 * kPostThreads) return launch_post_norm<T, 8, 1>(p, s);
    if (W % 8 == 0 && W > 8 * kPostThreads && W <= 2 * 8 * kPostThreads) return launch_post_norm<T, 8, 2>(p, s);
  }
  if (W % 4) return launch_post_norm<T, 1, 0>(p, s);
  if (W <= 4 * kPostThreads) return launch_post_norm<T, 4, 1>(p, s);
  if (W <= 4 * 4 * kPostThreads) return launch_post_norm<T, 4, 4>(p, s);
  return launch_post_norm<T, 4, 0>(p, s);
}

}  // namespace sb

using namespace sb;

// params: host PostNormParams; f32: activations and weights are fp32 (else bf16)
extern "C" int sb_post_norm_rows(const void* params, int f32, cudaStream_t stream) {
  const PostNormParams& p = *reinterpret_cast<const PostNormParams*>(params);
  if (p.rows <= 0) return 0;
  if (p.W < 1 || (p.ids && (!p.table || p.vocab < 1)) || (!p.ids && !p.post) || (p.ys && !(p.pair_slot && p.pair_w)) ||
      (p.y && p.slabs < 1))
    return -3;
  return f32 ? launch_post_norm_rows<float>(p, stream) : launch_post_norm_rows<__nv_bfloat16>(p, stream);
}
