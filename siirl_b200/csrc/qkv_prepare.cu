// What stands between the fused projection of an attention branch and its scores, one launch: sum of the projection's
// partial products, biases, RMS norms of queries and keys, rotation, append of keys and values to the paged cache
// (layout in win_params.h), queries in the activation format for the attention kernels, per-head output gates.  The
// branch's table of biases by distance is expanded from its buckets by blocks of its own.  Pooled runs of tokens (win_params.h):
// the block that appends the last token of a run writes the means of its keys and values (single tokens: pool_inline); the
// rows of a prompt portion meet in kv_pool_kernel, one launch later.
//
//   norm 0  none
//   norm 1  a whole projection (all heads at once) over its root mean square times a weight vector, before the rotation
//   norm 2  every head over its root mean square, no weight, after the rotation
//   norm 3  every head over its root mean square times one weight vector for all heads, before the rotation
//
// Rotation: pairs (i, i + half) of the first 2 * half dimensions of a head turn by position * f_i.  f_i comes as two
// floats (hi + lo) and the angle keeps its remainder, so the error does not grow with the position.
//
// qkv_prepare_units_kernel: a thread keeps its units of eight columns in registers as 32-bit floats and meets the other half of
// a rotated pair in shared memory; a block walks over rows, with the next row's loads in flight, one barrier per row.
// qkv_prepare_kernel: any sizes, one block per row, the row in shared memory.
#include <type_traits>

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
  float rot_mag;            // factor of cosines and sines
  int pool;                 // tokens per pooled run; 0: none
  const int* pool_table;    // [slots, pool_blocks] blocks of the pooled entries
  int pool_blocks, pool_inline;      // pool_inline: no two rows belong to one sequence
};
static_assert(sizeof(PrepareParams) == 240, "PrepareParams is mirrored from Python");

constexpr int kPrepBlk = 64;        // tokens per cache block
constexpr int kPrepThreads = 128;

// V columns of row t from `col` on, summed over the partial products, with the bias
template <typename T, int V>
__device__ __forceinline__ void prepare_fetch(const PrepareParams& p, int t, int col, float (&v)[V]) {
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
}

// this row's place in its cache block (head 0, keys), or null
template <typename T>
__device__ __forceinline__ T* prepare_block(const PrepareParams& p, int t, int& pos) {
  const int slot = p.seq_ids[t];
  pos = p.positions[t];
  if (slot < 0 || pos < 0 || pos / kPrepBlk >= p.max_blocks) return nullptr;
  const int blk = p.block_table[(size_t)slot * p.max_blocks + pos / kPrepBlk];
  if (blk < 0 || blk >= p.num_blocks) return nullptr;
  return reinterpret_cast<T*>(p.cache) + (size_t)blk * p.block_elems;
}

// Cosine and sine of a + lo.  Results that are rounded to 16 bits: a leaves its whole turns (2 pi as two floats, the first
// product exact in the fused multiply-add), the rest takes the special-function units (absolute error below 2^-21).
template <typename T>
__device__ __forceinline__ void turn_of(float a, float lo, float& c, float& s) {
  if constexpr (sizeof(T) == 2) {
    const float k = rintf(a * 0.15915494309189535f);
    const float r = fmaf(k, 1.7484556000744487e-07f, fmaf(k, -6.2831854820251465f, a)) + lo;
    s = __sinf(r);
    c = __cosf(r);
  } else {
    float s0, c0;
    sincosf(a, &s0, &c0);
    c = fmaf(-s0, lo, c0);
    s = fmaf(c0, lo, s0);
  }
}

// output gates of row t and the angles' cosines and sines.  PLANES: groups of eight angles as two planes of four
template <typename T, bool PLANES>
__device__ __forceinline__ void prepare_gates(const PrepareParams& p, int t, int pos, float* s_cos, float* s_sin) {
  if (p.g_off >= 0) {
    for (int h = threadIdx.x; h < p.Hq; h += blockDim.x) {
      float z[1];
      prepare_fetch<T, 1>(p, t, p.g_off + h, z);
      p.gate_out[(size_t)t * p.Hq + h] = 1.f / (1.f + expf(-z[0]));
    }
  }
  for (int i = threadIdx.x; i < p.half; i += blockDim.x) {
    const float n = (float)pos, a = n * p.freq[2 * i], lo = fmaf(n, p.freq[2 * i], -a) + n * p.freq[2 * i + 1];
    float s, c;
    turn_of<T>(a, lo, c, s);
    const int at = PLANES ? (i & 4 ? p.half / 2 : 0) + (i >> 3) * 4 + (i & 3) : i;
    s_cos[at] = c * p.rot_mag;
    s_sin[at] = s * p.rot_mag;
  }
}

// the run that ends at `pos` of the sequence in `slot`: means of its keys and values as the cache holds them, by all threads
// of a block.  V elements per access.
template <typename T, int V>
__device__ __forceinline__ void pool_run(const PrepareParams& p, int slot, int pos) {
  const int e = pos / p.pool, first = pos + 1 - p.pool;
  if (e / kPrepBlk >= p.pool_blocks || pos / kPrepBlk >= p.max_blocks) return;
  const int to = p.pool_table[(size_t)slot * p.pool_blocks + e / kPrepBlk];
  if (to < 0 || to >= p.num_blocks) return;
  const int* bt = p.block_table + (size_t)slot * p.max_blocks;
  T* cache = reinterpret_cast<T*>(p.cache);
  const int nk = p.Hkv * p.dk / V, n = p.Hkv * (p.dk + p.dv) / V;
  const float inv = 1.f / (float)p.pool;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const bool key = i < nk;
    const int d = key ? p.dk : p.dv, at = (key ? i : i - nk) * V, head = at / d;
    const size_t base = (key ? 0 : (size_t)p.Hkv * kPrepBlk * p.dk) + (size_t)head * kPrepBlk * d + (at - head * d);
    float sum[V] = {};
    // the blocks of a run are fetched one after the other, eight tokens of a block in flight
    for (int j = first; j <= pos;) {
      const int blk = bt[j / kPrepBlk], stop = min(pos + 1, (j / kPrepBlk + 1) * kPrepBlk);
      if (blk < 0 || blk >= p.num_blocks) {
        j = stop;
        continue;
      }
      const T* src = cache + (size_t)blk * p.block_elems + base;
#pragma unroll 8
      for (; j < stop; ++j) {
        float x[V];
        load_vec<T, V>(src + (size_t)(j % kPrepBlk) * d, x);
#pragma unroll
        for (int k = 0; k < V; ++k) sum[k] += x[k];
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k) sum[k] *= inv;
    store_vec<T, V>(cache + (size_t)to * p.block_elems + base + (size_t)(e % kPrepBlk) * d, sum);
  }
}

constexpr int kPoolThreads = 128;
// rows of a block: about one run ends among them
static int pool_rows(int pool) { return pool < 16 ? 16 : (pool < kPoolThreads ? pool : kPoolThreads); }

template <typename T, int V>
__global__ void __launch_bounds__(kPoolThreads) kv_pool_kernel(const __grid_constant__ PrepareParams p, int rows) {
  __shared__ int s_row[kPoolThreads], s_n;
  if (threadIdx.x == 0) s_n = 0;
  __syncthreads();
  const int t = blockIdx.x * rows + threadIdx.x;
  if ((int)threadIdx.x < rows && t < p.T) {
    const int slot = p.seq_ids[t], pos = p.positions[t];
    if (slot >= 0 && pos >= 0 && (pos + 1) % p.pool == 0) s_row[atomicAdd(&s_n, 1)] = t;
  }
  __syncthreads();
  for (int i = 0; i < s_n; ++i) pool_run<T, V>(p, p.seq_ids[s_row[i]], p.positions[s_row[i]]);
}

// blocks behind the `row_blocks` of the rows: the table of biases by distance
template <typename T>
__device__ __forceinline__ void prepare_table(const PrepareParams& p, int row_blocks) {
  const int n = p.Hq * p.rel_n, step = (gridDim.x - row_blocks) * blockDim.x;
  for (int i = (blockIdx.x - row_blocks) * blockDim.x + threadIdx.x; i < n; i += step) {
    const int h = i / p.rel_n, d = i - h * p.rel_n;
    p.rel_out[i] = to_float(reinterpret_cast<const T*>(p.rel)[(size_t)p.bucket[d] * p.Hq + h]);
  }
}

// eight elements as they lie in memory
template <typename T>
struct Unit {
  uint4 r[sizeof(T) / 2];
  __device__ __forceinline__ void load(const T* p) {
#pragma unroll
    for (int i = 0; i < (int)sizeof(T) / 2; ++i) r[i] = reinterpret_cast<const uint4*>(p)[i];
  }
  __device__ __forceinline__ void get(float (&x)[8]) const { load_vec<T, 8>(reinterpret_cast<const T*>(r), x); }
};

// eight floats as two planes of four: a warp's accesses fall on all banks evenly
__device__ __forceinline__ void store_planes(float* p, int plane, const float (&x)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  *reinterpret_cast<float4*>(p + plane) = make_float4(x[4], x[5], x[6], x[7]);
}
__device__ __forceinline__ void load_planes(const float* p, int plane, float (&x)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + plane);
  x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
  x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
}

// dk, dv and the rotated half are multiples of eight; a thread has U units of eight columns, the same in every row.  F32: the
// projection comes as 32-bit partial sums.
template <typename T, int U, bool F32>
__global__ void __launch_bounds__(512, U == 2 && !F32 ? 2 : 1) qkv_prepare_units_kernel(const __grid_constant__ PrepareParams p, int row_blocks) {
  extern __shared__ __align__(16) float sm[];
  if ((int)blockIdx.x >= row_blocks) return prepare_table<T>(p, row_blocks);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nq = p.Hq * p.dk / 8, nk = p.Hkv * p.dk / 8, nv = p.Hkv * p.dv / 8, per = p.dk / 8;      // units
  // two buffers: [nq + nk][8] weighted values (the norm's factor still to come), cosines, sines, sums of squares (norm 2)
  const int x_len = p.half ? 8 * (nq + nk) : 0, buf_len = (x_len + 2 * p.half + (p.norm >= 2 ? nq + nk : 0) + 7) / 8 * 8;
  const int plane = 4 * (nq + nk);
  const float inv_dk = 1.f / (float)p.dk;
  __shared__ float red[2][2][16];
  // heads whose units are a power of two lie in aligned lanes of one warp: their sums need no shared memory
  const bool in_warp = per <= 32 && (per & (per - 1)) == 0;
  int col[U], off[U], turn[U];        // column in x; place in the query row or in the cache block; first angle, + 1 << 16 in
                                      // the second half of a pair, -1: not rotated
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int i = tid + u * blockDim.x;
    col[u] = off[u] = 0;
    turn[u] = -1;
    if (i < nq + nk && i % per < p.half / 4) {
      const int at = i % per, half = p.half / 8;
      turn[u] = at < half ? 8 * at : 8 * (at - half) + (1 << 16);
    }
    if (i < nq) {
      col[u] = p.q_off + 8 * i;
      off[u] = 8 * i;
    } else if (i < nq + nk) {
      const int e = 8 * (i - nq), head = e / p.dk;
      col[u] = p.k_off + e;
      off[u] = head * kPrepBlk * p.dk + e - head * p.dk;
    } else if (i < nq + nk + nv) {
      const int e = 8 * (i - nq - nk), head = e / p.dv;
      col[u] = p.v_off + e;
      off[u] = p.Hkv * kPrepBlk * p.dk + head * kPrepBlk * p.dv + e - head * p.dv;
    }
  }
  Unit<T> weight[U];                  // of norms 1 and 3
  if (p.norm == 1 || p.norm == 3) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = tid + u * blockDim.x;
      if (i >= nq + nk) continue;
      weight[u].load(reinterpret_cast<const T*>(i < nq ? p.q_norm : p.k_norm) +
                     (p.norm == 3 ? 8 * (i % per) : 8 * (i < nq ? i : i - nq)));
    }
  }
  using X = typename std::conditional<F32, float, T>::type;
  Unit<X> next[U];
  auto fetch = [&](int t) {           // the first (or only) part of row t
#pragma unroll
    for (int u = 0; u < U; ++u) next[u].load(reinterpret_cast<const X*>(p.x) + (size_t)t * p.row_stride + col[u]);
  };
  // slot and position of the row after the next, block of the next
  auto place_of = [&](int t, int& slot, int& pos) {
    slot = pos = -1;
    if (t < p.T) {
      slot = p.seq_ids[t];
      pos = p.positions[t];
    }
  };
  auto block_of = [&](int slot, int pos) {
    return slot >= 0 && pos >= 0 && pos / kPrepBlk < p.max_blocks ? p.block_table[(size_t)slot * p.max_blocks + pos / kPrepBlk] : -1;
  };
  int t = blockIdx.x, slot0, pos0, slot1, pos1, buf = 0;
  fetch(t);
  place_of(t, slot0, pos0);
  place_of(t + row_blocks, slot1, pos1);
  int blk = block_of(slot0, pos0);
  for (; t < p.T; t += row_blocks, buf ^= 1) {
    float* s_x = sm + buf * buf_len;
    float* s_cos = s_x + x_len;
    float* s_sin = s_cos + p.half;
    float* s_part = s_sin + p.half;
    float v[U][8];
#pragma unroll
    for (int u = 0; u < U; ++u) next[u].get(v[u]);
    if (t + row_blocks < p.T) fetch(t + row_blocks);
    const int pos = pos0, place = pos % kPrepBlk;
    T* crow = blk >= 0 && blk < p.num_blocks ? reinterpret_cast<T*>(p.cache) + (size_t)blk * p.block_elems : nullptr;
    blk = block_of(slot1, pos1);
    pos0 = pos1;
    place_of(t + 2 * row_blocks, slot1, pos1);
    if constexpr (F32) {
      for (int s = 1; s < p.slabs; ++s)
#pragma unroll
        for (int u = 0; u < U; ++u) {
          float y[8];
          load_vec<float, 8>(reinterpret_cast<const float*>(p.x) + s * p.slab + (size_t)t * p.row_stride + col[u], y);
#pragma unroll
          for (int k = 0; k < 8; ++k) v[u][k] += y[k];
        }
    }
    prepare_gates<T, true>(p, t, pos, s_cos, s_sin);
    float ssq = 0.f, ssk = 0.f, own[U];      // own: squares of a unit's values before weights
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = tid + u * blockDim.x;
      own[u] = 0.f;
      if (p.bias && i < nq + nk + nv) {
        float b[8];
        load_vec<T, 8>(reinterpret_cast<const T*>(p.bias) + col[u], b);
#pragma unroll
        for (int k = 0; k < 8; ++k) v[u][k] += b[k];
      }
      if (i >= nq + nk) {
        if (i < nq + nk + nv && crow) store_vec<T, 8>(crow + off[u] + place * p.dv, v[u]);
        continue;
      }
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) ss = fmaf(v[u][k], v[u][k], ss);
      if (i < nq) ssq += ss;
      else ssk += ss;
      own[u] = ss;
      if (p.norm >= 2 && !in_warp) s_part[i] = ss;
      if (p.norm == 1 || p.norm == 3) {
        float w[8];
        weight[u].get(w);
#pragma unroll
        for (int k = 0; k < 8; ++k) v[u][k] *= w[k];
      }
      if (turn[u] >= 0) store_planes(s_x + 4 * i, plane, v[u]);
    }
    if (p.norm == 1) {
      ssq = warp_sum(ssq);
      ssk = warp_sum(ssk);
      if (lane == 0) {
        red[buf][0][warp] = ssq;
        red[buf][1][warp] = ssk;
      }
    }
    __syncthreads();      // the other buffer was last read before the barrier of the row before
    float fq = 1.f, fk = 1.f;
    if (p.norm == 1) {
      ssq = ssk = 0.f;
      for (int w = 0; w < (int)blockDim.x / 32; ++w) {
        ssq += red[buf][0][w];
        ssk += red[buf][1][w];
      }
      fq = rsqrtf(ssq / (float)(8 * nq) + p.eps);
      fk = rsqrtf(ssk / (float)(8 * nk) + p.eps);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = tid + u * blockDim.x;
      float f = i < nq ? fq : fk;
      if (p.norm >= 2) {
        float ss = 0.f;
        if (in_warp) {
          ss = own[u];
#pragma unroll
          for (int o = 16; o; o >>= 1)
            if (o < per) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        } else if (i < nq + nk) {
          const int h = i / per;
          for (int k = 0; k < per; ++k) ss += s_part[h * per + k];
        }
        f = rsqrtf(fmaf(ss, inv_dk, p.eps));
      }
      if (i >= nq + nk) continue;
      if (turn[u] >= 0) {
        const bool first = turn[u] < 1 << 16;
        const int r = (turn[u] & 0xffff) >> 1;
        float y[8], c[8], sn[8];
        load_planes(s_x + 4 * i + (first ? p.half : -p.half) / 2, plane, y);
        load_planes(s_cos + r, p.half / 2, c);
        load_planes(s_sin + r, p.half / 2, sn);
        const float fy = first ? -f : f;
#pragma unroll
        for (int k = 0; k < 8; ++k) v[u][k] = fmaf(v[u][k] * f, c[k], y[k] * fy * sn[k]);
      } else {
#pragma unroll
        for (int k = 0; k < 8; ++k) v[u][k] *= f;
      }
      if (i < nq) store_vec<T, 8>(reinterpret_cast<T*>(p.q_out) + (size_t)t * p.q_stride + off[u], v[u]);
      else if (crow) store_vec<T, 8>(crow + off[u] + place * p.dk, v[u]);
    }
    if (p.pool_inline && crow && (pos + 1) % p.pool == 0) {      // the same for the whole block
      __syncthreads();
      pool_run<T, 8>(p, p.seq_ids[t], pos);
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) qkv_prepare_kernel(const __grid_constant__ PrepareParams p, int row_blocks) {
  extern __shared__ float sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if ((int)blockIdx.x >= row_blocks) return prepare_table<T>(p, row_blocks);
  const int t = blockIdx.x;
  const int nq = p.Hq * p.dk, nk = p.Hkv * p.dk, nv = p.Hkv * p.dv;
  float* s_x = sm;                    // [nq + nk]
  float* s_cos = s_x + nq + nk;       // [half]
  float* s_sin = s_cos + p.half;
  __shared__ float red[2][kPrepThreads / 32];
  int pos;
  T* crow = prepare_block<T>(p, t, pos);
  const int place = pos % kPrepBlk;
  auto fetch = [&](int col, float (&v)[V]) {
    prepare_fetch<T, V>(p, t, col, v);
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
  prepare_gates<T, false>(p, t, pos, s_cos, s_sin);
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
    if (p.norm >= 2) {
      float ss = 0.f;
      for (int d = lane; d < p.dk; d += 32) ss = fmaf(x[d], x[d], ss);
      f = 1.f / sqrtf(warp_sum(ss) / (float)p.dk + p.eps);
    }
    const T* w = p.norm == 1 ? (is_q ? reinterpret_cast<const T*>(p.q_norm) + h * p.dk
                                     : reinterpret_cast<const T*>(p.k_norm) + kh * p.dk)
                             : (p.norm == 3 ? reinterpret_cast<const T*>(is_q ? p.q_norm : p.k_norm) : nullptr);
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
  if (p.pool_inline && crow && (pos + 1) % p.pool == 0) {
    __syncthreads();
    pool_run<T, V>(p, p.seq_ids[t], pos);
  }
}

using PrepareKernel = void (*)(PrepareParams, int);

static int prepare_configure(PrepareKernel kernel, size_t smem, size_t& configured) {
  if (smem <= configured) return 0;
  if (smem > 200 * 1024) return -3;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  configured = smem;
  return 0;
}

static int prepare_launch(PrepareKernel kernel, const PrepareParams& p, int row_blocks, int threads, size_t smem, cudaStream_t s) {
  int extra = 0;
  if (p.rel) {
    extra = (p.Hq * p.rel_n + 4 * threads - 1) / (4 * threads);
    if (extra > num_sms()) extra = num_sms();
  }
  kernel<<<row_blocks + extra, threads, smem, s>>>(p, row_blocks);
  return (int)cudaGetLastError();
}

template <typename T, int V>
static int launch_prepare(const PrepareParams& p, cudaStream_t s) {
  static size_t configured = 48 * 1024;
  const size_t smem = ((size_t)(p.Hq + p.Hkv) * p.dk + 2 * (size_t)p.half) * 4;
  const int r = prepare_configure(qkv_prepare_kernel<T, V>, smem, configured);
  return r ? r : prepare_launch(qkv_prepare_kernel<T, V>, p, p.T, kPrepThreads, smem, s);
}

template <typename T, int U, bool F32>
static int launch_prepare_units(const PrepareParams& p, cudaStream_t s) {
  auto kernel = qkv_prepare_units_kernel<T, U, F32>;
  const int qk = (p.Hq + p.Hkv) * p.dk, units = (qk + p.Hkv * p.dv) / 8;
  const int threads = ((units + U - 1) / U + 31) / 32 * 32;
  const size_t smem = 8 * (((size_t)(p.half ? qk : 0) + 2 * (size_t)p.half + (p.norm >= 2 ? qk / 8 : 0) + 7) / 8 * 8);
  static size_t configured = 48 * 1024;
  const int r = prepare_configure(kernel, smem, configured);
  if (r) return r;
  int blocks = 1;
  if (p.T > num_sms()) {
    cudaError_t e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&blocks, kernel, threads, smem);
    if (e != cudaSuccess) return (int)e;
    if (blocks < 1) blocks = 1;
  }
  blocks *= num_sms();
  return prepare_launch(kernel, p, p.T < blocks ? p.T : blocks, threads, smem, s);
}

template <typename T>
static int launch_prepare_units(const PrepareParams& p, int units, cudaStream_t s) {
  if (p.x_f32) return units <= 2 * 512 ? launch_prepare_units<T, 2, true>(p, s) : launch_prepare_units<T, 4, true>(p, s);
  return units <= 2 * 512 ? launch_prepare_units<T, 2, false>(p, s) : launch_prepare_units<T, 4, false>(p, s);
}

}  // namespace sb

using namespace sb;

// params: host PrepareParams; f32: activations, weights and cache are fp32 (else bf16)
extern "C" int sb_qkv_prepare(const void* params, int f32, cudaStream_t stream) {
  const PrepareParams& p = *reinterpret_cast<const PrepareParams*>(params);
  if (p.T <= 0) return 0;
  if (p.Hkv < 1 || p.Hq % p.Hkv || p.dk < 1 || p.dv < 1 || 2 * p.half > p.dk || p.slabs < 1 || (p.slabs > 1 && !p.x_f32) ||
      ((p.norm == 1 || p.norm == 3) && !(p.q_norm && p.k_norm)) || (p.half && !p.freq) || (p.g_off >= 0 && !p.gate_out) ||
      (p.rel && !(p.bucket && p.rel_out)) || p.norm < 0 || p.norm > 3 || p.pool < 0 || (p.pool && !(p.pool_table && p.pool_blocks > 0)))
    return -3;
  const int V = f32 ? 4 : 8;
  const bool vec = p.dk % V == 0 && p.dv % V == 0 && p.row_stride % V == 0 && p.slab % V == 0 && p.q_off % V == 0 &&
                   p.k_off % V == 0 && p.v_off % V == 0 && p.q_stride % V == 0 && p.block_elems % V == 0;
  const int units = ((p.Hq + p.Hkv) * p.dk + p.Hkv * p.dv) / 8;
  if (vec && p.dk % 8 == 0 && p.dv % 8 == 0 && p.half % 8 == 0 && units <= 4 * 512) {
    return f32 ? launch_prepare_units<float>(p, units, stream) : launch_prepare_units<__nv_bfloat16>(p, units, stream);
  }
  if (f32) return vec ? launch_prepare<float, 4>(p, stream) : launch_prepare<float, 1>(p, stream);
  return vec ? launch_prepare<__nv_bfloat16, 8>(p, stream) : launch_prepare<__nv_bfloat16, 1>(p, stream);
}

// The pooled runs that end among the rows of prompt portions (their keys and values are in the cache): same arguments
extern "C" int sb_kv_pool(const void* params, int f32, cudaStream_t stream) {
  const PrepareParams& p = *reinterpret_cast<const PrepareParams*>(params);
  if (p.T <= 0) return 0;
  if (p.pool < 1 || !p.pool_table || p.pool_blocks < 1 || p.Hkv < 1 || p.dk < 1 || p.dv < 1) return -3;
  const int V = f32 ? 4 : 8;
  const bool vec = p.dk % V == 0 && p.dv % V == 0 && p.block_elems % V == 0;
  const int rows = pool_rows(p.pool), grid = (p.T + rows - 1) / rows;
  if (f32) {
    if (vec) kv_pool_kernel<float, 4><<<grid, kPoolThreads, 0, stream>>>(p, rows);
    else kv_pool_kernel<float, 1><<<grid, kPoolThreads, 0, stream>>>(p, rows);
  } else {
    if (vec) kv_pool_kernel<__nv_bfloat16, 8><<<grid, kPoolThreads, 0, stream>>>(p, rows);
    else kv_pool_kernel<__nv_bfloat16, 1><<<grid, kPoolThreads, 0, stream>>>(p, rows);
  }
  return (int)cudaGetLastError();
}
