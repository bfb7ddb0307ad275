// Row operations of decoders whose residual stream is kept in 32-bit floats, and a plain SIMT matrix product for the
// shapes and number formats the tensor-core GEMM does not take.
//
//   embed_scaled       h[t] = table[id[t]] * scale                               (fp32 stream)
//   add_norm           h += delta;  y = norm(h) * w                              (layer norm or RMS norm, one launch)
//   stream_rows        h += mult * sum of two sublayer results, each times a sigmoid gate, then h / rms(h)  (one launch);
//                      or h = sum of partial products + vector (entry of a loop's pass), then h / rms(h); or h as two rows
//   gated_act          y = act(gate) * up   for a fused projection [gate | up]   (SiLU, tanh-form or exact GELU, squared relu)
//   scaled_act         y = act(gain * x)    of a column range
//   bias_act           y = act(sum of partial products + bias), xIELU with its two learned numbers among the activations
//   token_gate         y = gelu_tanh(sum of partial products) * columns of an embedding table's row
//   softcap            z = cap * tanh(z / cap) in place on fp32 logits
//   gemm_simt          C[M, N] = A[M, K] B[N, K]^T with fp32 accumulation on the FMA pipes: fp32 models (true 32-bit
//                      products) and bf16 operands whose row pitch TMA cannot address (not a multiple of 16 bytes)
//
// Templates: T is the activation / weight format (bf16 or fp32); V elements per access (4, or 1 for odd widths).
#include <type_traits>

#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"

namespace sb {

template <typename T, int V>
__global__ void embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                                    float* __restrict__ h, int T_, int W, int vocab, float scale) {
  const int nv = W / V;
  const long long total = (long long)T_ * nv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / nv), c = (int)(i % nv) * V;
    long long id = ids[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    float x[V];
    load_vec<T, V>(table + (size_t)id * W + c, x);
#pragma unroll
    for (int k = 0; k < V; ++k) x[k] *= scale;
    store_vec<float, V>(h + (size_t)t * W + c, x);
  }
}

constexpr int kRowThreads = 256;

__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = red[0];
#pragma unroll
  for (int i = 1; i < kRowThreads / 32; ++i) t += red[i];
  return t;
}

// CH register chunks of V elements per thread hold the row (CH = 0: the row is re-read from memory)
template <typename T, int V, int CH>
__global__ void __launch_bounds__(kRowThreads)
add_norm_kernel(float* __restrict__ h, const T* __restrict__ delta, const T* __restrict__ w, T* __restrict__ y, int rows,
                int W, float eps, int layer_norm) {
  __shared__ float red[kRowThreads / 32];
  const int nv = W / V;
  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    float* hr = h + (size_t)row * W;
    float x[CH > 0 ? CH : 1][V];
    float s = 0.f;
    auto fetch = [&](int vi, float (&v)[V]) {
      load_vec<float, V>(hr + (size_t)vi * V, v);
      if (delta) {
        float d[V];
        load_vec<T, V>(delta + (size_t)row * W + (size_t)vi * V, d);
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] += d[k];
        store_vec<float, V>(hr + (size_t)vi * V, v);
      }
    };
    auto each = [&](auto&& fn) {
      if constexpr (CH > 0) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
          const int vi = threadIdx.x + c * kRowThreads;
          if (vi < nv) fn(vi, x[c]);
        }
      } else {
        for (int vi = threadIdx.x; vi < nv; vi += kRowThreads) {
          load_vec<float, V>(hr + (size_t)vi * V, x[0]);   // written by this same thread below
          fn(vi, x[0]);
        }
      }
    };
    if constexpr (CH > 0) {
      each([&](int vi, float (&v)[V]) { fetch(vi, v); });
    } else {
      for (int vi = threadIdx.x; vi < nv; vi += kRowThreads) fetch(vi, x[0]);
    }
    float mean = 0.f;
    if (layer_norm) {
      each([&](int, float (&v)[V]) {
#pragma unroll
        for (int k = 0; k < V; ++k) s += v[k];
      });
      mean = row_sum(s, red) / (float)W;
    }
    float ss = 0.f;
    each([&](int, float (&v)[V]) {
#pragma unroll
      for (int k = 0; k < V; ++k) ss += (v[k] - mean) * (v[k] - mean);
    });
    const float rstd = 1.f / sqrtf(row_sum(ss, red) / (float)W + eps);
    each([&](int vi, float (&v)[V]) {
      float wv[V], o[V];
      load_vec<T, V>(w + (size_t)vi * V, wv);
#pragma unroll
      for (int k = 0; k < V; ++k) o[k] = (v[k] - mean) * rstd * wv[k];
      store_vec<T, V>(y + (size_t)row * W + (size_t)vi * V, o);
    });
  }
}

__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return 0.5f * z * (1.f + tanhf(u));
}

// z Phi(z) with the normal distribution function from formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical
// Functions (|error of erf| <= 1.5e-7), evaluated on the side where nothing cancels: for results that are rounded to 16 bits
__device__ __forceinline__ float gelu_erf_fast(float z) {
  const float x = fabsf(z) * 0.7071067811865476f;
  const float t = __fdividef(1.f, fmaf(0.3275911f, x, 1.f));
  float q = fmaf(1.061405429f, t, -1.453152027f);
  q = fmaf(q, t, 1.421413741f);
  q = fmaf(q, t, -0.284496736f);
  q = fmaf(q, t, 0.254829592f);
  q *= 0.5f * t * __expf(-x * x);       // Phi(-|z|)
  return z * (z < 0.f ? q : 1.f - q);
}

template <int ACT, typename T>      // 0 SiLU, 1 tanh-form GELU, 2 exact GELU, 3 square of relu; T: the format of the result
__device__ __forceinline__ float activate(float z) {
  if constexpr (ACT == 3) {
    z = fmaxf(z, 0.f);
    return z * z;
  }
  if constexpr (ACT == 0 && sizeof(T) == 4) return z / (1.f + expf(-z));
  if constexpr (ACT == 1) return gelu_tanh_f(z);
  if constexpr (ACT == 2 && sizeof(T) == 2) return gelu_erf_fast(z);
  if constexpr (ACT == 2) return 0.5f * z * (1.f + erff(z * 0.7071067811865476f));
  return z / (1.f + __expf(-z));
}

// sigmoid of a gate whose product is added to a 32-bit stream (T = float: every step in full precision)
template <typename T>
__device__ __forceinline__ float gate_sigmoid(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  return 1.f / (1.f + expf(-z));
}

template <typename T, int V, int ACT>
__global__ void gated_act_kernel(const T* __restrict__ gu, T* __restrict__ out, long long rows, int I,
                                 const int* __restrict__ used) {
  const int nv = I / V;
  const long long total = rows * nv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / nv;
    if (used && used[t] < 0) continue;      // padding row of an expert's segment
    const int c = (int)(i % nv) * V;
    float g[V], u[V];
    load_vec<T, V>(gu + t * 2 * I + c, g);
    load_vec<T, V>(gu + t * 2 * I + I + c, u);
#pragma unroll
    for (int k = 0; k < V; ++k) g[k] = activate<ACT, T>(g[k]) * u[k];
    store_vec<T, V>(out + t * I + c, g);
  }
}

template <typename T, int V, int ACT>
__global__ void scaled_act_kernel(const T* __restrict__ x, long long stride, const T* __restrict__ gain, T* __restrict__ out,
                                  long long rows, int I) {
  // a thread keeps its columns and walks down the rows, four loads in flight
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= I) return;
  const float f = gain ? to_float(*gain) : 1.f;
  const long long step = gridDim.y;
  for (long long t = blockIdx.y; t < rows; t += 4 * step) {
    float v[4][V];
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (t + u * step < rows) load_vec<T, V>(x + (t + u * step) * stride + c, v[u]);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (t + u * step >= rows) break;
#pragma unroll
      for (int k = 0; k < V; ++k) v[u][k] = activate<ACT, T>(f * v[u][k]);
      store_vec<T, V>(out + (t + u * step) * I + c, v[u]);
    }
  }
}

// act of the sum of fp32 partial products [slabs, rows, I or 2 I] (GATED: act(first half) * second half), bf16 result
template <int V, int ACT, bool GATED>
__global__ void partial_act_kernel(const float* __restrict__ x, long long slab, int slabs, __nv_bfloat16* __restrict__ out,
                                   long long rows, int I) {
  const int nv = I / V, pitch = GATED ? 2 * I : I;
  const long long total = rows * nv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / nv;
    const int c = (int)(i % nv) * V;
    float g[V] = {}, u[V] = {};
    const float* p = x + t * pitch + c;
    for (int s = 0; s < slabs; ++s, p += slab) {
      float a[V];
      load_vec<float, V>(p, a);
#pragma unroll
      for (int k = 0; k < V; ++k) g[k] += a[k];
      if constexpr (GATED) {
        load_vec<float, V>(p + I, a);
#pragma unroll
        for (int k = 0; k < V; ++k) u[k] += a[k];
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k) g[k] = activate<ACT, __nv_bfloat16>(g[k]) * (GATED ? u[k] : 1.f);
    store_vec<__nv_bfloat16, V>(out + t * I + c, g);
  }
}

// Two learned numbers: softplus(p) z^2 + z / 2 on the right of zero, (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 on the left
struct Xielu {
  float right = 0.f, left = 0.f;
  Xielu() = default;
  template <typename T>
  __device__ __forceinline__ explicit Xielu(const T* n)
      : right(softplus(to_float(n[0]))), left(0.5f + softplus(to_float(n[1]))) {}
  static __device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
  // the result is rounded to T: next to zero (where e^z - 1 - z cancels) its first terms, z^2 (1/2 + z/6 + z^2/24 + z^3/120)
  template <typename T>
  __device__ __forceinline__ float operator()(float z) const {
    if constexpr (sizeof(T) == 4) {
      return z > 0.f ? fmaf(right * z, z, 0.5f * z) : fmaf(left, expm1f(z) - z, 0.5f * z);
    } else {
      const float zz = z * z;
      const float near = zz * fmaf(z, fmaf(z, fmaf(z, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f);
      const float far = __expf(z) - 1.f - z;
      return fmaf(z > 0.f ? right : left, z > 0.f ? zz : (z > -0.25f ? near : far), 0.5f * z);
    }
  }
};

// ACT 4: xIELU.  XT: format of x (partial sums: fp32); T: of bias, numbers and result
template <typename XT, typename T, int V, int ACT>
__global__ void bias_act_kernel(const XT* __restrict__ x, long long slab, int slabs, const T* __restrict__ bias,
                                const T* __restrict__ numbers, T* __restrict__ out, long long rows, int I,
                                const int* __restrict__ used) {
  // a thread keeps its columns and walks down the rows, four loads in flight
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= I) return;
  float b[V] = {};
  if (bias) load_vec<T, V>(bias + c, b);
  Xielu xi;
  if constexpr (ACT == 4) xi = Xielu(numbers);
  const long long step = gridDim.y;
  for (long long t = blockIdx.y; t < rows; t += 4 * step) {
    float v[4][V];
    bool on[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const long long r = t + u * step;
      on[u] = r < rows && !(used && used[r] < 0);
      if (on[u]) load_vec<XT, V>(x + r * I + c, v[u]);
    }
    for (int s = 1; s < slabs; ++s) {
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (!on[u]) continue;
        float a[V];
        load_vec<XT, V>(x + s * slab + (t + u * step) * I + c, a);
#pragma unroll
        for (int k = 0; k < V; ++k) v[u][k] += a[k];
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (!on[u]) continue;
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const float z = v[u][k] + b[k];
        if constexpr (ACT == 4) v[u][k] = xi.template operator()<T>(z);
        else v[u][k] = activate<ACT, T>(z);
      }
      store_vec<T, V>(out + (t + u * step) * I + c, v[u]);
    }
  }
}

template <typename XT, typename T, int V>
__global__ void token_gate_kernel(const XT* __restrict__ z, long long slab, int slabs, const long long* __restrict__ ids,
                                  const T* __restrict__ table, long long pitch, int vocab, int column, int width,
                                  T* __restrict__ out, int rows, int I) {
  const int nv = I / V;
  const long long total = (long long)rows * nv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / nv), c = (int)(i % nv) * V;
    long long id = ids[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    float g[V], e[V];
    load_vec<XT, V>(z + (size_t)t * I + c, g);
    const T* row = table + id * pitch + column + c;
    if constexpr (V == 1) e[0] = c < width ? to_float(*row) : 0.f;
    else load_vec<T, V>(row, e);      // width is a multiple of V
    for (int s = 1; s < slabs; ++s) {
      float a[V];
      load_vec<XT, V>(z + s * slab + (size_t)t * I + c, a);
#pragma unroll
      for (int k = 0; k < V; ++k) g[k] += a[k];
    }
#pragma unroll
    for (int k = 0; k < V; ++k) g[k] = gelu_tanh_f(g[k]) * e[k];
    store_vec<T, V>(out + (size_t)t * I + c, g);
  }
}

// mirrored by ctypes structures in ops/rows.py
struct StreamSub {
  const void* y;            // [slabs, T or 2 T, W] partial sums (fp32), or one tensor in the activation format
  long long slab;
  int slabs, y_f32;
  const void* gate;         // pre-activations of the gate, or null
  long long gate_stride;
  const void* bias;         // [W], or null
  const void* gain;         // one number, or null
};
struct StreamParams {
  float* h;                 // [rows, W]
  int rows, W;
  float mult, eps;
  int n_sub, enter;         // enter: h is replaced by sub[0] + sub[1] + step
  StreamSub sub[2];
  const void* step;         // [W]
  int pair, split;          // pair: sub[0] has 2 rows per row of h; split: out is h as two rows of the format, [2 rows, W]
  const void* weight;       // one number, or null
  void* out;                // [rows, W] (or [2 rows, W]) in the activation format
};
static_assert(sizeof(StreamParams) == 176, "StreamParams is mirrored from Python");

// CH register chunks of V elements per thread hold the row (CH = 0: the row is re-read from memory).  WHOLE: the update of
// a prompt, both results one gated tensor each in the activation format, all loads issued before the first use.
template <typename T, int V, int CH, bool WHOLE = false>
__global__ void __launch_bounds__(kRowThreads) stream_rows_kernel(const __grid_constant__ StreamParams p) {
  __shared__ float red[kRowThreads / 32];
  const int W = p.W, nv = W / V;
  float gain[2];
#pragma unroll
  for (int j = 0; j < 2; ++j) gain[j] = p.sub[j].gain ? to_float(*reinterpret_cast<const T*>(p.sub[j].gain)) : 1.f;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    float* hr = p.h + (size_t)row * W;
    T* o0 = reinterpret_cast<T*>(p.out) + (size_t)row * W;
    float x[CH > 0 ? CH : 1][V];
    // sum of the slabs of sublayer j at vector vi of row r
    auto add_slabs = [&](const StreamSub& s, int r, int vi, float (&v)[V]) {
      const size_t at = (size_t)r * W + (size_t)vi * V;
      for (int k = 0; k < s.slabs; ++k) {
        float y[V];
        if (s.y_f32) load_vec<float, V>(reinterpret_cast<const float*>(s.y) + k * s.slab + at, y);
        else load_vec<T, V>(reinterpret_cast<const T*>(s.y) + k * s.slab + at, y);
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] += y[i];
      }
    };
    auto fetch = [&](int vi, float (&v)[V]) {
      const size_t c = (size_t)vi * V;
      if constexpr (WHOLE) {
        float y[2][V], g[2][V], b[2][V];
        load_vec<float, V>(hr + c, v);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          load_vec<T, V>(reinterpret_cast<const T*>(p.sub[j].y) + (size_t)row * W + c, y[j]);
          load_vec<T, V>(reinterpret_cast<const T*>(p.sub[j].gate) + row * p.sub[j].gate_stride + c, g[j]);
          load_vec<T, V>(reinterpret_cast<const T*>(p.sub[j].bias) + c, b[j]);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) {
          const float add = y[0][i] * gate_sigmoid<T>(fmaf(gain[0], g[0][i], b[0][i])) +
                            y[1][i] * gate_sigmoid<T>(fmaf(gain[1], g[1][i], b[1][i]));
          v[i] = fmaf(p.mult, add, v[i]);
        }
      } else if (p.enter) {
        load_vec<T, V>(reinterpret_cast<const T*>(p.step) + c, v);
        add_slabs(p.sub[1], row, vi, v);
        add_slabs(p.sub[0], row, vi, v);
        if (p.pair) add_slabs(p.sub[0], row + p.rows, vi, v);
      } else {
        load_vec<float, V>(hr + c, v);
        float add[V] = {};
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          if (j >= p.n_sub) break;
          const StreamSub& s = p.sub[j];
          float y[V] = {};
          add_slabs(s, row, vi, y);
          if (s.gate) {
            float g[V], b[V] = {};
            load_vec<T, V>(reinterpret_cast<const T*>(s.gate) + row * s.gate_stride + c, g);
            if (s.bias) load_vec<T, V>(reinterpret_cast<const T*>(s.bias) + c, b);
#pragma unroll
            for (int i = 0; i < V; ++i) y[i] *= gate_sigmoid<T>(fmaf(gain[j], g[i], b[i]));
          }
#pragma unroll
          for (int i = 0; i < V; ++i) add[i] += y[i];
        }
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = fmaf(p.mult, add[i], v[i]);
      }
      if (p.enter || p.n_sub) store_vec<float, V>(hr + c, v);
      if (p.split) {
        store_vec<T, V>(o0 + c, v);
        if constexpr (sizeof(T) == 2) {
          float lo[V];
#pragma unroll
          for (int i = 0; i < V; ++i) lo[i] = v[i] - __bfloat162float(__float2bfloat16(v[i]));
          store_vec<T, V>(o0 + (size_t)p.rows * W + c, lo);
        }
      }
    };
    if constexpr (CH > 0) {
#pragma unroll
      for (int c = 0; c < CH; ++c) {
        const int vi = threadIdx.x + c * kRowThreads;
        if (vi < nv) fetch(vi, x[c]);
      }
    } else {
      for (int vi = threadIdx.x; vi < nv; vi += kRowThreads) fetch(vi, x[0]);
    }
    if (p.split) continue;
    auto each = [&](auto&& fn) {
      if constexpr (CH > 0) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
          const int vi = threadIdx.x + c * kRowThreads;
          if (vi < nv) fn(vi, x[c]);
        }
      } else {
        for (int vi = threadIdx.x; vi < nv; vi += kRowThreads) {
          load_vec<float, V>(hr + (size_t)vi * V, x[0]);   // written by this same thread above
          fn(vi, x[0]);
        }
      }
    };
    float ss = 0.f;
    each([&](int, float (&v)[V]) {
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(v[k], v[k], ss);
    });
    float f = 1.f / sqrtf(row_sum(ss, red) / (float)W + p.eps);
    if (p.weight) f *= to_float(*reinterpret_cast<const T*>(p.weight));
    each([&](int vi, float (&v)[V]) {
      float o[V];
#pragma unroll
      for (int k = 0; k < V; ++k) o[k] = v[k] * f;
      store_vec<T, V>(o0 + (size_t)vi * V, o);
    });
  }
}

template <int V>
__global__ void softcap_kernel(float* __restrict__ z, long long n, float cap) {
  const float inv = 1.f / cap;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n / V; i += (long long)gridDim.x * blockDim.x) {
    float x[V];
    load_vec<float, V>(z + i * V, x);
#pragma unroll
    for (int k = 0; k < V; ++k) x[k] = cap * tanhf(x[k] * inv);
    store_vec<float, V>(z + i * V, x);
  }
}

// 64 x 64 output tile per 256 threads, 4 x 4 values each, contraction in steps of 16 through shared memory.
// GROUPED: rows are slots of experts, 128-row blocks of one expert each (tile_group, -1: unused block); a slot's row of A is
// a_row[slot] (-1: zeros) when given, and B holds one matrix per expert, b_group elements apart.
template <typename TI, typename TO, bool GROUPED = false>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const TI* __restrict__ A, const TI* __restrict__ B, TO* __restrict__ C, int M, int N, int K,
                 long long lda, long long ldb, long long ldc, const int* __restrict__ tile_group = nullptr,
                 const int* __restrict__ a_row = nullptr, long long b_group = 0) {
  __shared__ float sa[16][68], sb_[16][68];
  __shared__ int s_row[64];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  if constexpr (GROUPED) {
    const int g = tile_group[m0 / 128];
    if (g < 0) return;
    B += (size_t)g * b_group;
    if (threadIdx.x < 64) {
      const int m = m0 + threadIdx.x;
      s_row[threadIdx.x] = m < M ? (a_row ? a_row[m] : m) : -1;
    }
    __syncthreads();
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i >> 4, k = i & 15;
      const int row = GROUPED ? s_row[r] : (m0 + r < M ? m0 + r : -1);
      sa[k][r] = (row >= 0 && k0 + k < K) ? to_float(A[(size_t)row * lda + k0 + k]) : 0.f;
      sb_[k][r] = (n0 + r < N && k0 + k < K) ? to_float(B[(size_t)(n0 + r) * ldb + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = sa[k][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = sb_[k][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) C[(size_t)m * ldc + n] = from_float<TO>(acc[i][j]);
    }
}

static int grid_for(long long total, int threads) {
  long long b = (total + threads - 1) / threads;
  const long long cap = (long long)num_sms() * 8;
  return (int)(b < 1 ? 1 : (b > cap ? cap : b));
}

template <typename T>
static int launch_add_norm(float* h, const T* delta, const T* w, T* y, int rows, int W, float eps, int ln, cudaStream_t s) {
  const int grid = rows < num_sms() * 8 ? rows : num_sms() * 8;
  if (W % 4) {
    add_norm_kernel<T, 1, 0><<<grid, kRowThreads, 0, s>>>(h, delta, w, y, rows, W, eps, ln);
  } else if (W <= 4 * kRowThreads) {
    add_norm_kernel<T, 4, 1><<<grid, kRowThreads, 0, s>>>(h, delta, w, y, rows, W, eps, ln);
  } else if (W <= 4 * 4 * kRowThreads) {
    add_norm_kernel<T, 4, 4><<<grid, kRowThreads, 0, s>>>(h, delta, w, y, rows, W, eps, ln);
  } else {
    add_norm_kernel<T, 4, 0><<<grid, kRowThreads, 0, s>>>(h, delta, w, y, rows, W, eps, ln);
  }
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_stream_rows(const StreamParams& p, cudaStream_t s) {
  const int grid = p.rows < num_sms() * 8 ? p.rows : num_sms() * 8, W = p.W;
  auto takes = [&](int v) {      // accesses of v elements of the activation format
    bool ok = W % v == 0;
    for (int j = 0; j < 2; ++j)
      ok = ok && p.sub[j].gate_stride % v == 0 && (uintptr_t)p.sub[j].gate % (v * sizeof(T)) == 0;
    return ok;
  };
  bool whole = !p.enter && p.n_sub == 2;
  for (int j = 0; j < 2; ++j)
    whole = whole && p.sub[j].gate && p.sub[j].bias && p.sub[j].slabs == 1 && (p.sub[j].y_f32 != 0) == (sizeof(T) == 4);
  if (sizeof(T) == 2 && takes(8) && whole && W <= 2 * 8 * kRowThreads) {
    if (W <= 8 * kRowThreads) stream_rows_kernel<T, 8, 1, true><<<grid, kRowThreads, 0, s>>>(p);
    else stream_rows_kernel<T, 8, 2, true><<<grid, kRowThreads, 0, s>>>(p);
  } else if (sizeof(T) == 2 && takes(8) && W <= 2 * 8 * kRowThreads) {
    if (W <= 8 * kRowThreads) stream_rows_kernel<T, 8, 1><<<grid, kRowThreads, 0, s>>>(p);
    else stream_rows_kernel<T, 8, 2><<<grid, kRowThreads, 0, s>>>(p);
  } else if (!takes(4)) {
    stream_rows_kernel<T, 1, 0><<<grid, kRowThreads, 0, s>>>(p);
  } else if (W <= 4 * kRowThreads) {
    stream_rows_kernel<T, 4, 1><<<grid, kRowThreads, 0, s>>>(p);
  } else if (W <= 2 * 4 * kRowThreads) {
    stream_rows_kernel<T, 4, 2><<<grid, kRowThreads, 0, s>>>(p);
  } else {
    stream_rows_kernel<T, 4, 0><<<grid, kRowThreads, 0, s>>>(p);
  }
  return (int)cudaGetLastError();
}

template <typename T, int V>
static int launch_gated_act(const T* gu, T* out, long long rows, int I, int act, const int* used, int grid, cudaStream_t s) {
  if (act == 0) gated_act_kernel<T, V, 0><<<grid, 256, 0, s>>>(gu, out, rows, I, used);
  else if (act == 1) gated_act_kernel<T, V, 1><<<grid, 256, 0, s>>>(gu, out, rows, I, used);
  else if (act == 2) gated_act_kernel<T, V, 2><<<grid, 256, 0, s>>>(gu, out, rows, I, used);
  else gated_act_kernel<T, V, 3><<<grid, 256, 0, s>>>(gu, out, rows, I, used);
  return (int)cudaGetLastError();
}

template <typename XT, typename T, int V>
static int launch_bias_act(const XT* x, long long slab, int slabs, const T* bias, const T* numbers, T* out, long long rows,
                           int I, int act, const int* used, cudaStream_t s) {
  const int threads = I / V >= 256 ? 256 : 64, cols = (I / V + threads - 1) / threads;
  long long y = (long long)num_sms() * (2048 / threads) / cols + 1;
  if (y > rows) y = rows;
  const dim3 grid(cols, (unsigned)(y > 65535 ? 65535 : y));
  auto launch = [&](auto kernel) { kernel<<<grid, threads, 0, s>>>(x, slab, slabs, bias, numbers, out, rows, I, used); };
  switch (act) {
    case 0: launch(bias_act_kernel<XT, T, V, 0>); break;
    case 1: launch(bias_act_kernel<XT, T, V, 1>); break;
    case 2: launch(bias_act_kernel<XT, T, V, 2>); break;
    case 3: launch(bias_act_kernel<XT, T, V, 3>); break;
    default: launch(bias_act_kernel<XT, T, V, 4>); break;
  }
  return (int)cudaGetLastError();
}

template <typename T, int V>
static int launch_scaled_act(const T* x, long long stride, const T* gain, T* out, long long rows, int I, int act,
                             cudaStream_t s) {
  const int cols = (I / V + 255) / 256;
  long long y = num_sms() * 8 / cols + 1;      // about eight blocks per SM
  if (y > rows) y = rows;
  const dim3 grid(cols, (unsigned)(y > 65535 ? 65535 : y));
  if (act == 0) scaled_act_kernel<T, V, 0><<<grid, 256, 0, s>>>(x, stride, gain, out, rows, I);
  else if (act == 1) scaled_act_kernel<T, V, 1><<<grid, 256, 0, s>>>(x, stride, gain, out, rows, I);
  else if (act == 2) scaled_act_kernel<T, V, 2><<<grid, 256, 0, s>>>(x, stride, gain, out, rows, I);
  else scaled_act_kernel<T, V, 3><<<grid, 256, 0, s>>>(x, stride, gain, out, rows, I);
  return (int)cudaGetLastError();
}

}  // namespace sb

using namespace sb;

// f32: 1 when tables, activations and weights are fp32, 0 for bf16 (the stream `h` is always fp32)
extern "C" int sb_embed_scaled(const long long* ids, const void* table, float* h, int T, int W, int vocab, float scale,
                               int f32, cudaStream_t stream) {
  if (T == 0) return 0;
  const int grid = grid_for((long long)T * W / 4, 256);
  if (f32) {
    if (W % 4 == 0) embed_scaled_kernel<float, 4><<<grid, 256, 0, stream>>>(ids, (const float*)table, h, T, W, vocab, scale);
    else embed_scaled_kernel<float, 1><<<grid, 256, 0, stream>>>(ids, (const float*)table, h, T, W, vocab, scale);
  } else {
    using B = __nv_bfloat16;
    if (W % 4 == 0) embed_scaled_kernel<B, 4><<<grid, 256, 0, stream>>>(ids, (const B*)table, h, T, W, vocab, scale);
    else embed_scaled_kernel<B, 1><<<grid, 256, 0, stream>>>(ids, (const B*)table, h, T, W, vocab, scale);
  }
  return (int)cudaGetLastError();
}

// h [rows, W] fp32 is updated in place (+= delta when given); y = norm(h) * w in the activation format
extern "C" int sb_add_norm(float* h, const void* delta, const void* w, void* y, int rows, int W, float eps,
                           int layer_norm, int f32, cudaStream_t stream) {
  if (rows == 0) return 0;
  if (f32)
    return launch_add_norm<float>(h, (const float*)delta, (const float*)w, (float*)y, rows, W, eps, layer_norm, stream);
  return launch_add_norm<__nv_bfloat16>(h, (const __nv_bfloat16*)delta, (const __nv_bfloat16*)w, (__nv_bfloat16*)y, rows,
                                        W, eps, layer_norm, stream);
}

// act: 0 SiLU, 1 tanh-form GELU, 2 exact GELU, 3 square of relu; gu [rows, 2 I] -> out [rows, I]; used: rows with a
// negative entry are left out (null: none)
extern "C" int sb_gated_act(const void* gu, void* out, long long rows, int I, int act, const int* used, int f32,
                            cudaStream_t stream) {
  if (rows == 0) return 0;
  if (act < 0 || act > 3) return -3;
  const int V = f32 ? 4 : 8;
  const int grid = grid_for(rows * I / (I % V ? 1 : V), 256);
  using B = __nv_bfloat16;
  if (f32)
    return I % 4 == 0 ? launch_gated_act<float, 4>((const float*)gu, (float*)out, rows, I, act, used, grid, stream)
                      : launch_gated_act<float, 1>((const float*)gu, (float*)out, rows, I, act, used, grid, stream);
  return I % 8 == 0 ? launch_gated_act<B, 8>((const B*)gu, (B*)out, rows, I, act, used, grid, stream)
                    : launch_gated_act<B, 1>((const B*)gu, (B*)out, rows, I, act, used, grid, stream);
}

// x: columns of rows `stride` apart -> out [rows, I]; gain: one number or null
extern "C" int sb_scaled_act(const void* x, long long stride, const void* gain, void* out, long long rows, int I, int act,
                             int f32, cudaStream_t stream) {
  if (rows == 0 || I == 0) return 0;
  if (act < 0 || act > 3) return -3;
  const int V = f32 ? 4 : 8;
  const bool vec = I % V == 0 && stride % V == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)out & 15) == 0;
  using B = __nv_bfloat16;
  if (f32)
    return vec ? launch_scaled_act<float, 4>((const float*)x, stride, (const float*)gain, (float*)out, rows, I, act, stream)
               : launch_scaled_act<float, 1>((const float*)x, stride, (const float*)gain, (float*)out, rows, I, act, stream);
  return vec ? launch_scaled_act<B, 8>((const B*)x, stride, (const B*)gain, (B*)out, rows, I, act, stream)
             : launch_scaled_act<B, 1>((const B*)x, stride, (const B*)gain, (B*)out, rows, I, act, stream);
}

// params: host StreamParams
extern "C" int sb_stream_rows(const void* params, int f32, cudaStream_t stream) {
  const StreamParams& p = *reinterpret_cast<const StreamParams*>(params);
  if (p.rows <= 0) return 0;
  if (p.n_sub < 0 || p.n_sub > 2 || (p.enter && p.n_sub != 2)) return -3;
  return f32 ? launch_stream_rows<float>(p, stream) : launch_stream_rows<__nv_bfloat16>(p, stream);
}

extern "C" int sb_softcap(float* z, long long n, float cap, cudaStream_t stream) {
  if (n == 0) return 0;
  if (!(cap > 0.f)) return -3;
  if (n % 4 == 0 && ((uintptr_t)z & 15) == 0) softcap_kernel<4><<<grid_for(n / 4, 256), 256, 0, stream>>>(z, n, cap);
  else softcap_kernel<1><<<grid_for(n, 256), 256, 0, stream>>>(z, n, cap);
  return (int)cudaGetLastError();
}

// in_f32: operands fp32 (else bf16); out_f32: result fp32 (else bf16)
extern "C" int sb_gemm_simt(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb,
                            long long ldc, int in_f32, int out_f32, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if ((M + 63) / 64 > 65535) return -3;
  const dim3 grid((N + 63) / 64, (M + 63) / 64);
  using H = __nv_bfloat16;
  if (in_f32 && out_f32)
    gemm_simt_kernel<float, float><<<grid, 256, 0, stream>>>((const float*)A, (const float*)B, (float*)C, M, N, K, lda, ldb, ldc);
  else if (!in_f32 && out_f32)
    gemm_simt_kernel<H, float><<<grid, 256, 0, stream>>>((const H*)A, (const H*)B, (float*)C, M, N, K, lda, ldb, ldc);
  else if (!in_f32)
    gemm_simt_kernel<H, H><<<grid, 256, 0, stream>>>((const H*)A, (const H*)B, (H*)C, M, N, K, lda, ldb, ldc);
  else
    return -2;
  return (int)cudaGetLastError();
}

// Products of expert slots: C[slot] = A[a_row[slot] or slot] B[expert of the slot]^T, fp32 operands and results or bf16
extern "C" int sb_gemm_simt_grouped(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb,
                                    long long ldc, const int* tile_group, const int* a_row, long long b_group, int f32,
                                    cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if (M % 128 || M / 64 > 65535 || !tile_group) return -3;
  const dim3 grid((N + 63) / 64, M / 64);
  using H = __nv_bfloat16;
  if (f32)
    gemm_simt_kernel<float, float, true><<<grid, 256, 0, stream>>>((const float*)A, (const float*)B, (float*)C, M, N, K, lda,
                                                                   ldb, ldc, tile_group, a_row, b_group);
  else
    gemm_simt_kernel<H, H, true><<<grid, 256, 0, stream>>>((const H*)A, (const H*)B, (H*)C, M, N, K, lda, ldb, ldc,
                                                           tile_group, a_row, b_group);
  return (int)cudaGetLastError();
}

// act of the sum of partial products; I a multiple of 4.  gated: x [slabs, rows, 2 I], else [slabs, rows, I]
extern "C" int sb_partial_act(const float* x, long long slab, int slabs, void* out, long long rows, int I, int act, int gated,
                              cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (I % 4 || slab % 4 || slabs < 1 || act < 0 || act > 3) return -3;
  const int grid = grid_for(rows * I / 4, 256);
  auto launch = [&](auto kernel) { kernel<<<grid, 256, 0, stream>>>(x, slab, slabs, (__nv_bfloat16*)out, rows, I); };
  if (gated) {
    if (act == 0) launch(partial_act_kernel<4, 0, true>);
    else if (act == 1) launch(partial_act_kernel<4, 1, true>);
    else if (act == 2) launch(partial_act_kernel<4, 2, true>);
    else launch(partial_act_kernel<4, 3, true>);
  } else {
    if (act == 0) launch(partial_act_kernel<4, 0, false>);
    else if (act == 1) launch(partial_act_kernel<4, 1, false>);
    else if (act == 2) launch(partial_act_kernel<4, 2, false>);
    else launch(partial_act_kernel<4, 3, false>);
  }
  return (int)cudaGetLastError();
}

// act (4: xIELU with two numbers) of the sum of x [slabs, rows, I] (fp32, or one slab in the activation format) plus bias;
// rows with a negative entry in `used` are left out
extern "C" int sb_bias_act(const void* x, long long slab, int slabs, int x_f32, const void* bias, const void* numbers, void* out,
                           long long rows, int I, int act, const int* used, int f32, cudaStream_t stream) {
  if (rows <= 0 || I <= 0) return 0;
  if (act < 0 || act > 4 || (act == 4 && !numbers) || slabs < 1 || (f32 && !x_f32) || (slabs > 1 && !x_f32)) return -3;
  const bool aligned = (((uintptr_t)x | (uintptr_t)out | (uintptr_t)bias) & 15) == 0;
  using B = __nv_bfloat16;
  auto run = [&](auto* xp, auto* op, auto vec) -> int {
    using T = std::remove_pointer_t<decltype(op)>;
    using XT = std::remove_const_t<std::remove_pointer_t<decltype(xp)>>;
    constexpr int V = decltype(vec)::value;
    return launch_bias_act<XT, T, V>(xp, slab, slabs, (const T*)bias, (const T*)numbers, op, rows, I, act, used, stream);
  };
  if (f32) {
    if (I % 4 == 0 && aligned) return run((const float*)x, (float*)out, std::integral_constant<int, 4>());
    return run((const float*)x, (float*)out, std::integral_constant<int, 1>());
  }
  if (x_f32) {
    if (I % 4 == 0 && aligned) return run((const float*)x, (B*)out, std::integral_constant<int, 4>());
    return run((const float*)x, (B*)out, std::integral_constant<int, 1>());
  }
  if (I % 8 == 0 && aligned) return run((const B*)x, (B*)out, std::integral_constant<int, 8>());
  return run((const B*)x, (B*)out, std::integral_constant<int, 1>());
}

// gelu_tanh of the sum of z [slabs, rows, I] times table[ids, column .. + width] (rows `pitch` apart); columns past `width`
// become zero
extern "C" int sb_token_gate(const void* z, long long slab, int slabs, int z_f32, const long long* ids, const void* table,
                             long long pitch, int vocab, int column, int width, void* out, int rows, int I, int f32,
                             cudaStream_t stream) {
  if (rows <= 0 || I <= 0) return 0;
  if (slabs < 1 || (f32 && !z_f32) || (slabs > 1 && !z_f32) || width < 1 || width > I || column < 0 || column + width > pitch)
    return -3;
  using B = __nv_bfloat16;
  const int V = f32 || z_f32 ? 4 : 8;
  const bool vec = width == I && I % V == 0 && column % V == 0 && pitch % V == 0 &&
                   (((uintptr_t)z | (uintptr_t)table | (uintptr_t)out) & 15) == 0;
  const int grid = grid_for((long long)rows * I / (vec ? V : 1), 128);
#define SB_GATE(XT, T, VV) \
  token_gate_kernel<XT, T, VV><<<grid, 128, 0, stream>>>((const XT*)z, slab, slabs, ids, (const T*)table, pitch, vocab, column, width, (T*)out, rows, I)
  if (f32) {
    if (vec) SB_GATE(float, float, 4);
    else SB_GATE(float, float, 1);
  } else if (z_f32) {
    if (vec) SB_GATE(float, B, 4);
    else SB_GATE(float, B, 1);
  } else {
    if (vec) SB_GATE(B, B, 8);
    else SB_GATE(B, B, 1);
  }
#undef SB_GATE
  return (int)cudaGetLastError();
}
