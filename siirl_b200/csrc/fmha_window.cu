// Attention of prompt portions against the paged cache with a sliding window, kept first tokens or pooled runs before it, and
// a linear distance bias (see win_params.h), and the cache append for heads whose key and value widths differ.
//
// The portion's keys and values are appended to the cache first; a query tile then walks the cache blocks in which any
// of its rows sees a key: the blocks of the kept first tokens or of the pooled entries, then those of the window.  Whole prompts, later portions
// and reused prefixes take the same path, and blocks that left every window are never touched.  Keys and values may also
// lie in packed rows (latent attention expands them from its cache), and the result may be gated.
//
//   window_prefill_kernel   bf16, dk and dv multiples of 8 up to 256: 128 query rows of one head per CTA, S = Q K^T and
//                           O += P V on tcgen05 with accumulators in TMEM; one cache block is one K/V tile, fetched by
//                           TMA straight from the paged cache (columns past dk / dv are filled with zeros)
//                           (two forms: linear bias or pooled runs; soft cap and a bias table by distance)
//   window_simt_kernel      any sizes, bf16 or fp32, one CTA per (row, head): the 32-bit path, and odd widths
#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"
#include "win_params.h"

namespace sb {

constexpr int kWBlk = 64;

template <typename T, int V>
__global__ void kv_append_split_kernel(WinParams p) {
  const int nk = p.Hkv * p.dk / V, nv = p.Hkv * p.dv / V;
  const long long total = (long long)p.T * (nk + nv);
  for (long long idx = blockIdx.x * (long long)blockDim.x + threadIdx.x; idx < total;
       idx += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(idx / (nk + nv));
    int r = (int)(idx % (nk + nv));
    const int slot = p.seq_ids[t], pos = p.positions[t];
    if (slot < 0 || pos < 0 || pos / kWBlk >= p.max_blocks) continue;
    const int blk = p.block_table[(size_t)slot * p.max_blocks + pos / kWBlk];
    if (blk < 0 || blk >= p.num_blocks) continue;
    const bool is_v = r >= nk;
    if (is_v) r -= nk;
    const int d = is_v ? p.dv : p.dk;
    const int head = r * V / d, e = r * V % d;
    const T* src = reinterpret_cast<const T*>(p.x) + (size_t)t * p.row_stride + (is_v ? p.v_off : p.k_off) + (size_t)r * V;
    T* dst = reinterpret_cast<T*>(p.cache) + (size_t)blk * p.block_elems + (is_v ? (size_t)p.Hkv * kWBlk * p.dk : 0) +
             ((size_t)head * kWBlk + pos % kWBlk) * d + e;
    float x[V];
    load_vec<T, V>(src, x);
    store_vec<T, V>(dst, x);
  }
}

constexpr int kSimtThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kSimtThreads) window_simt_kernel(WinParams p) {
  extern __shared__ float sm[];
  float* sq = sm;                      // [dk]
  float* sp = sq + p.dk;               // [128] weights of the current keys
  float* so = sp + kSimtThreads;       // [dv]
  __shared__ float red[8];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int slot = p.seq_ids[t], i = p.positions[t];
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.out_stride + p.out_off + (size_t)h * p.dv;
  if (slot < 0 || i < 0) {
    for (int d = tid; d < p.dv; d += kSimtThreads) out[d] = from_float<T>(0.f);
    return;
  }
  const int kvh = h / (p.Hq / p.Hkv);
  const float slope = p.bias_exp > 0.f ? exp2f(-p.bias_exp * (h + 1) / p.Hq) : 0.f;
  const T* q = reinterpret_cast<const T*>(p.x) + (size_t)t * p.row_stride + p.q_off + (size_t)h * p.dk;
  const float gain = p.gain ? to_float(*reinterpret_cast<const T*>(p.gain)) : 1.f;
  for (int d = tid; d < p.dk; d += kSimtThreads) sq[d] = to_float(q[d]) * gain;
  for (int d = tid; d < p.dv; d += kSimtThreads) so[d] = 0.f;
  // the visible keys are 0 .. first - 1 (tokens, or pooled entries) and lo .. i
  int first = 0, lo = 0;
  if (p.pool > 0) {
    first = pooled_entries(i, p.window, p.pool);
    lo = max(0, i - p.window + 1);
  } else if (p.window > 0) {
    first = min(p.keep_first, i + 1);
    lo = max(first, i - p.window + 1);
  }
  const int n = first + (i + 1 - lo);
  const int* bt = p.block_table + (size_t)slot * p.max_blocks;
  const int* pt = p.pool > 0 ? p.pool_table + (size_t)slot * p.pool_blocks : bt;
  const int pt_blocks = p.pool > 0 ? p.pool_blocks : p.max_blocks;
  const T* cache = reinterpret_cast<const T*>(p.cache);
  auto row_of = [&](int v, bool value) -> const T* {
    const int j = v < first ? v : lo + v - first;
    const int blk = v < first ? (j / kWBlk < pt_blocks ? pt[j / kWBlk] : -1) : (j / kWBlk < p.max_blocks ? bt[j / kWBlk] : -1);
    if (blk < 0 || blk >= p.num_blocks) return nullptr;
    const size_t base = (size_t)blk * p.block_elems;
    return value && p.kv_mode != kLatent
               ? cache + base + (size_t)p.Hkv * kWBlk * p.dk + ((size_t)kvh * kWBlk + j % kWBlk) * p.dv
               : cache + base + ((size_t)kvh * kWBlk + j % kWBlk) * p.dk;
  };
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  for (int v0 = 0; v0 < n; v0 += kSimtThreads) {
    const int v = v0 + tid;
    float s = -INFINITY;
    if (v < n) {
      const T* k = row_of(v, false);
      if (k) {
        float acc = 0.f;
        for (int d = 0; d < p.dk; ++d) acc = fmaf(sq[d], to_float(k[d]), acc);
        const int j = v < first ? v : lo + v - first;
        s = acc * p.scale - slope * (float)(i - j);
        if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
        if (p.rel) s += p.rel[(size_t)h * p.rel_n + min((long long)(i - j), p.rel_n - 1)];
      }
    }
    float mx = warp_max(s);
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float mn = fmaxf(m, mx);
    const float w = s == -INFINITY ? 0.f : expf(s - mn);
    const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
    sp[tid] = w;
    const float ws = warp_sum(w);
    if (lane == 0) red[4 + warp] = ws;
    __syncthreads();
    l = l * alpha + red[4] + red[5] + red[6] + red[7];
    m = mn;
    const int cnt = min(kSimtThreads, n - v0);
    for (int d = tid; d < p.dv; d += kSimtThreads) {
      float acc = so[d] * alpha;
      for (int c = 0; c < cnt; ++c) {
        const T* vr = row_of(v0 + c, true);
        if (vr) acc = fmaf(sp[c], to_float(vr[d]), acc);
      }
      so[d] = acc;
    }
    __syncthreads();
  }
  if (p.sink_w) l += expf(to_float(reinterpret_cast<const T*>(p.sink_w)[h]) - m);
  else if (p.sink) l += expf(-m);
  float inv = l > 0.f ? p.out_scale / l : 0.f;
  if (p.head_gate) inv *= p.head_gate[(size_t)t * p.Hq + h];
  for (int d = tid; d < p.dv; d += kSimtThreads) out[d] = from_float<T>(so[d] * inv);
}

// ---------------------------------------------------------------------------------------
// tensor-core prefill
// ---------------------------------------------------------------------------------------
struct WinSmem {
  int q_bytes, k_bytes, v_bytes, k_off, v_off, p_off, bar_off, total;
  __host__ __device__ WinSmem(int ck, int cv) {      // 64-column chunks of the key and value widths
    q_bytes = ck * 128 * 128;
    k_bytes = ck * kWBlk * 128;
    v_bytes = cv * kWBlk * 128;
    k_off = q_bytes;
    v_off = k_off + 2 * k_bytes;
    p_off = v_off + 2 * v_bytes;
    bar_off = p_off + 128 * kWBlk * 2;
    total = bar_off + 96;
  }
};

// cache blocks a query tile at positions q0 .. q1 visits: `sinks` blocks from 0 (of the tokens, or of the pooled entries), then
// blocks w0 .. of the window
__host__ __device__ inline void win_blocks(int q0, int q1, int window, int keep_first, int pool, int& sinks, int& w0, int& n) {
  const int last = q1 / kWBlk;
  if (pool > 0) {
    sinks = (pooled_entries(q1, window, pool) + kWBlk - 1) / kWBlk;
    w0 = q0 - window + 1 > 0 ? (q0 - window + 1) / kWBlk : 0;
  } else if (window <= 0) {
    sinks = 0;
    w0 = 0;
  } else {
    sinks = (keep_first + kWBlk - 1) / kWBlk;
    if (sinks > last + 1) sinks = last + 1;
    const int lo = q0 - window + 1;
    w0 = lo > 0 ? lo / kWBlk : 0;
    if (w0 < sinks) w0 = sinks;
  }
  n = sinks + (last + 1 > w0 ? last + 1 - w0 : 0);
}

// Warp 4 fetches and issues: S(j + 1) = Q K(j + 1)^T goes ahead of O += P(j) V(j), into the other half of a double-buffered S,
// so the scores of the next tile are computed while warps 0 - 3 (one row per thread) are in the soft-max of this one.  A key
// tile is given back when its scores are done, a value tile one step later.  The running maximum is only raised when it grows
// by more than 2^8.  TABLE: soft-capped scores and / or a bias table by distance instead of the linear bias.
template <bool TABLE>
__global__ void __launch_bounds__(160, 2)
window_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_v, WinParams p, const int* __restrict__ tile_row,
                      const int* __restrict__ tile_rows, const int* __restrict__ tile_pos,
                      const int* __restrict__ tile_slot, uint32_t tmem_cols, int* status) {
  const int ck = (p.dk + 63) / 64, cv = (p.dv + 63) / 64;
  const int k_steps = (p.dk + 15) / 16, vn = (p.dv + 15) / 16 * 16;
  const WinSmem L(ck, cv);
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw;
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0) atomicCAS(status, 0, (int)kStatusBadArgument);
    return;
  }
  uint8_t* sQ = smem;
  uint8_t* sK = smem + L.k_off;
  uint8_t* sV = smem + L.v_off;
  uint8_t* sP = smem + L.p_off;
  uint64_t* bar_q = reinterpret_cast<uint64_t*>(smem + L.bar_off);
  uint64_t* bar_k = bar_q + 1;      // [2] key tile has arrived
  uint64_t* bar_v = bar_q + 3;      // [2] value tile has arrived
  uint64_t* bar_s = bar_q + 5;      // [2] scores are in TMEM
  uint64_t* bar_p = bar_q + 7;      // weights are in shared memory (and the scores have been read)
  uint64_t* bar_o = bar_q + 8;      // O holds this tile
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar_q + 9);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int tile = blockIdx.x, h = blockIdx.y;
  const int row0 = tile_row[tile], nrows = tile_rows[tile], q0 = tile_pos[tile], slot = tile_slot[tile];
  const int kvh = h / (p.Hq / p.Hkv);
  int sinks, w0, n_tiles;
  win_blocks(q0, q0 + nrows - 1, p.window, p.keep_first, p.pool, sinks, w0, n_tiles);
  const bool packed = p.kv_mode == kPackedRows;
  const int* bt = p.block_table + (size_t)(packed ? 0 : slot) * p.max_blocks;
  const bool pool = !TABLE && p.pool > 0;
  const int* pt = pool ? p.pool_table + (size_t)slot * p.pool_blocks : nullptr;
  auto block_of = [&](int j) { return j < sinks ? j : w0 + j - sinks; };

  if (tid == 0) {
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
    for (int i = 0; i < 9; ++i) mbar_init(&bar_q[i], i == 7 ? 4 : 1);
    fence_barrier_init();
  }
  if (warp == 4) {
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 128;
  bool ok = true;

  if (warp == 4) {
    // ------------------------------ copies and MMAs (the warp stays converged, lane 0 issues) ------------------------------
    const uint32_t leader = lane == 0;
    int k_loads = 0, v_loads = 0;
    // packed rows: head kvh, rows from the block on; those past the sequence are hidden by causality, past the end zeros
    auto load = [&](const CUtensorMap* map, uint8_t* dst, int bytes, int chunks, uint64_t* bar, int j) {
      const int lb = block_of(j);
      int blk;
      if (pt && j < sinks) blk = lb < p.pool_blocks ? pt[lb] : 0;
      else blk = packed ? slot + lb * kWBlk : (lb < p.max_blocks ? bt[lb] : 0);
      if (!packed && (blk < 0 || blk >= p.num_blocks)) blk = 0;      // never inside the visible range of a well-formed table
      const int mid = packed ? kvh : kvh * kWBlk;
      if (leader) {
        mbar_arrive_expect_tx(bar, (uint32_t)bytes);
        for (int c = 0; c < chunks; ++c) tma_load_3d(dst + c * 8192, map, bar, c * 64, mid, blk);
      }
    };
    auto load_k = [&](int j) {
      load(&map_k, sK + (j & 1) * L.k_bytes, L.k_bytes, ck, &bar_k[j & 1], j);
      ++k_loads;
    };
    auto load_v = [&](int j) {
      load(&map_v, sV + (j & 1) * L.v_bytes, L.v_bytes, cv, &bar_v[j & 1], j);
      ++v_loads;
    };
    auto wait = [&](uint64_t* bar, uint32_t parity) {
      return __all_sync(0xffffffffu, mbar_wait(bar, parity, status, kStatusTimeoutMma));
    };
    if (leader) {
      mbar_arrive_expect_tx(bar_q, (uint32_t)L.q_bytes);
      for (int c = 0; c < ck; ++c) tma_load_3d(sQ + c * 16384, &map_q, bar_q, c * 64, h, row0);
    }
    for (int j = 0; j < 2 && j < n_tiles; ++j) {
      load_k(j);
      load_v(j);
    }
    const uint32_t idesc_s = umma_idesc_bf16(128, kWBlk, 0, 0);
    const uint32_t idesc_o = umma_idesc_bf16(128, vn, 0, 1);
    const uint64_t dq = umma_smem_desc(smem_u32(sQ), 16, 1024), dk0 = umma_smem_desc(smem_u32(sK), 16, 1024);
    const uint64_t dp = umma_smem_desc(smem_u32(sP), 16, 1024), dv0 = umma_smem_desc(smem_u32(sV), 8192, 1024);
    const uint32_t k_step = (uint32_t)L.k_bytes >> 4, v_step = (uint32_t)L.v_bytes >> 4;
    auto scores = [&](int j) {
      uint64_t da = dq, db = dk0 + (j & 1) * k_step;
      const uint32_t d = tmem_s + (j & 1) * 64;
      int left = k_steps;
#pragma unroll 1
      for (int c = 0; c < ck; ++c, da += 1024, db += 512, left -= 4) {
        umma_bf16_ss_if(leader, d, da, db, idesc_s, c ? 1u : 0u);
        if (left > 1) umma_bf16_ss_if(leader, d, da + 2, db + 2, idesc_s, 1u);
        if (left > 2) umma_bf16_ss_if(leader, d, da + 4, db + 4, idesc_s, 1u);
        if (left > 3) umma_bf16_ss_if(leader, d, da + 6, db + 6, idesc_s, 1u);
      }
      umma_commit_if(leader, &bar_s[j & 1]);
    };
    ok = wait(bar_q, 0) && wait(&bar_k[0], 0);
    if (ok) {
      tc_fence_after();
      scores(0);
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      if (j + 1 < n_tiles) {
        ok = wait(&bar_k[(j + 1) & 1], ((j + 1) >> 1) & 1);
        if (!ok) break;
        tc_fence_after();
        scores(j + 1);
      }
      ok = wait(&bar_s[j & 1], (j >> 1) & 1);
      if (!ok) break;
      if (j + 2 < n_tiles) load_k(j + 2);
      if (j > 0) {
        ok = wait(bar_o, (j - 1) & 1);
        if (!ok) break;
        if (j + 1 < n_tiles) load_v(j + 1);
      }
      ok = wait(bar_p, j & 1) && wait(&bar_v[j & 1], (j >> 1) & 1);
      if (!ok) break;
      tc_fence_after();
      const uint64_t db = dv0 + (j & 1) * v_step;
      umma_bf16_ss_if(leader, tmem_o, dp, db, idesc_o, j ? 1u : 0u);
      umma_bf16_ss_if(leader, tmem_o, dp + 2, db + 128, idesc_o, 1u);
      umma_bf16_ss_if(leader, tmem_o, dp + 4, db + 256, idesc_o, 1u);
      umma_bf16_ss_if(leader, tmem_o, dp + 6, db + 384, idesc_o, 1u);
      umma_commit_if(leader, bar_o);
    }
    if (!ok) {      // bounded: let the copies in flight land before shared memory is given back
      mbar_wait(bar_q, 0, nullptr, 0);
      for (int st = 0; st < 2; ++st) {
        const int nk = (k_loads + 1 - st) / 2, nv = (v_loads + 1 - st) / 2;
        if (nk) mbar_wait(&bar_k[st], (nk - 1) & 1, nullptr, 0);
        if (nv) mbar_wait(&bar_v[st], (nv - 1) & 1, nullptr, 0);
      }
    }
  } else {
    // ------------------------------ soft-max and result ------------------------------
    const uint32_t lane_off = (uint32_t)(warp * 32) << 16;
    const int qpos = q0 + tid;
    const float gain = p.gain ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(p.gain)) : 1.f;
    const float scale_log2 = p.scale * gain * 1.4426950408889634f;
    const float slope_log2 =
        p.bias_exp > 0.f ? exp2f(-p.bias_exp * (float)(h + 1) / (float)p.Hq) * 1.4426950408889634f : 0.f;
    const ScoreCap cap(p.softcap > 0.f ? p.softcap : 1.f, p.scale * gain);
    const float* rel = TABLE && p.rel ? p.rel + (size_t)h * p.rel_n : nullptr;
    const int rel_last = (int)p.rel_n - 1;
    const float rel_far = rel ? __ldg(rel + rel_last) * 1.4426950408889634f : 0.f;
    const int pool_q0 = pooled_entries(q0, p.window, p.pool), pool_n = pooled_entries(qpos, p.window, p.pool);
    float m_ref = -INFINITY, l_run = 0.f;

    for (int j = 0; j < n_tiles; ++j) {
      if (!__all_sync(0xffffffffu, mbar_wait(&bar_s[j & 1], (j >> 1) & 1, status, kStatusTimeoutEpilogue))) {
        ok = false;
        break;
      }
      tc_fence_after();
      const int kv0 = block_of(j) * kWBlk;
      float sv[kWBlk];
      {
        uint32_t r0[32], r1[32];
        tmem_ld_32x32(tmem_s + (j & 1) * 64 + lane_off, r0);
        tmem_ld_32x32(tmem_s + (j & 1) * 64 + lane_off + 32, r1);
        tmem_ld_wait();
        if constexpr (TABLE) {
          if (p.softcap > 0.f) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              sv[i] = cap(__uint_as_float(r0[i]));
              sv[32 + i] = cap(__uint_as_float(r1[i]));
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              sv[i] = __uint_as_float(r0[i]) * scale_log2;
              sv[32 + i] = __uint_as_float(r1[i]) * scale_log2;
            }
          }
          const int d0 = qpos - kv0;      // distance of the tile's first key
          if (rel && q0 - (kv0 + kWBlk - 1) >= rel_last) {      // the whole tile is at least as far as the last entry
#pragma unroll
            for (int i = 0; i < kWBlk; ++i) sv[i] += rel_far;
          } else if (rel && q0 >= kv0 + kWBlk - 1 && q0 + 127 - kv0 <= rel_last) {      // the whole tile lies inside the table
            const float* at = rel + d0 - (kWBlk - 1);
#pragma unroll
            for (int i = 0; i < kWBlk; ++i) sv[i] = fmaf(__ldg(at + (kWBlk - 1 - i)), 1.4426950408889634f, sv[i]);
          } else if (rel) {
#pragma unroll
            for (int i = 0; i < kWBlk; ++i)
              sv[i] = fmaf(__ldg(rel + min(max(d0 - i, 0), rel_last)), 1.4426950408889634f, sv[i]);
          }
        } else {
          // score in units of log 2, distance bias included: s * scale - slope * (i - j)
          const float b0 = slope_log2 * (float)(kv0 - qpos);
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            sv[i] = fmaf(__uint_as_float(r0[i]), scale_log2, fmaf(slope_log2, (float)i, b0));
            sv[32 + i] = fmaf(__uint_as_float(r1[i]), scale_log2, fmaf(slope_log2, (float)(32 + i), b0));
          }
        }
      }
      // every row of the tile sees every key of the block when the block lies behind q0 and, with a window, inside the
      // last row's window or among the kept tokens
      if (pool && j < sinks) {      // entries kv0 .. of the pooled runs
        if (kv0 + kWBlk > pool_q0) {
#pragma unroll
          for (int i = 0; i < kWBlk; ++i)
            if (kv0 + i >= pool_n) sv[i] = -INFINITY;
        }
      } else if (!(kv0 + kWBlk - 1 <= q0 &&
                   (p.window <= 0 || q0 + nrows - 1 - kv0 < p.window || kv0 + kWBlk <= p.keep_first))) {
#pragma unroll
        for (int i = 0; i < kWBlk; ++i) {
          const int kp = kv0 + i;
          if (!(kp <= qpos && (p.window <= 0 || qpos - kp < p.window || kp < p.keep_first))) sv[i] = -INFINITY;
        }
      }
      float m4[4] = {sv[0], sv[1], sv[2], sv[3]};
#pragma unroll
      for (int i = 4; i < kWBlk; ++i) m4[i & 3] = fmaxf(m4[i & 3], sv[i]);
      const float m_tile = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
      float alpha = 1.f;
      const bool raise = m_tile > m_ref + 8.f;
      if (raise) {
        alpha = exp2f(m_ref - m_tile);      // 0 the first time
        l_run *= alpha;
        m_ref = m_tile;
      }
      const bool rescale = j > 0 && __any_sync(0xffffffffu, raise);
      const float m_safe = m_ref == -INFINITY ? 0.f : m_ref;
      float s4[4] = {};
      uint32_t pk[kWBlk / 2];
#pragma unroll
      for (int i = 0; i < kWBlk; i += 2) {
        const float p0 = fast_exp2(sv[i] - m_safe), p1 = fast_exp2(sv[i + 1] - m_safe);
        s4[(i >> 1) & 3] += p0 + p1;
        pk[i / 2] = pack_bf16x2(p0, p1);
      }
      l_run += (s4[0] + s4[1]) + (s4[2] + s4[3]);
      // the tile before has left the weights' buffer and is in O
      if (j > 0 && !__all_sync(0xffffffffu, mbar_wait(bar_o, (j - 1) & 1, status, kStatusTimeoutEpilogue))) {
        ok = false;
        break;
      }
      if (rescale) {
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < (vn + 31) / 32; ++c) {
          uint32_t r[32];
          tmem_ld_32x32(tmem_o + lane_off + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
          tmem_st_32x32(tmem_o + lane_off + c * 32, r);
        }
        tmem_st_wait();
      }
      {
        uint8_t* prow = sP + tid * 128;
#pragma unroll
        for (int piece = 0; piece < 8; ++piece) {
          uint4 v = make_uint4(pk[piece * 4], pk[piece * 4 + 1], pk[piece * 4 + 2], pk[piece * 4 + 3]);
          *reinterpret_cast<uint4*>(prow + ((piece ^ (tid & 7)) << 4)) = v;
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_p);
    }
    if (ok)
      ok = __all_sync(0xffffffffu, mbar_wait(bar_o, (n_tiles - 1) & 1, status, kStatusTimeoutEpilogue));
    if (ok) {
      tc_fence_after();
      const bool row_valid = tid < nrows;
      if (p.sink_w) l_run += exp2f(fmaf(__bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.sink_w)[h]), 1.4426950408889634f, -m_ref));
      else if (p.sink) l_run += exp2f(-m_ref);
      float inv_l = l_run > 0.f ? p.out_scale / l_run : 0.f;
      if (p.head_gate && row_valid) inv_l *= p.head_gate[(size_t)(row0 + tid) * p.Hq + h];
      __nv_bfloat16* orow = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(row0 + (row_valid ? tid : 0)) * p.out_stride +
                            p.out_off + (size_t)h * p.dv;
      const __nv_bfloat16* grow = reinterpret_cast<const __nv_bfloat16*>(p.gate) +
                                  (size_t)(row0 + (row_valid ? tid : 0)) * p.gate_stride + (size_t)h * p.dv;
#pragma unroll 1
      for (int c = 0; c < (vn + 31) / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(tmem_o + lane_off + c * 32, r);
        tmem_ld_wait();
        if (row_valid) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            if (c * 32 + g * 8 >= p.dv) break;
            float o[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) o[i] = __uint_as_float(r[g * 8 + i]) * inv_l;
            if (p.gate) {
              float z[8];
              load_vec<__nv_bfloat16, 8>(grow + c * 32 + g * 8, z);
#pragma unroll
              for (int i = 0; i < 8; ++i) o[i] = __fdividef(o[i], 1.f + __expf(-gain * z[i]));
            }
            store_vec<__nv_bfloat16, 8>(orow + c * 32 + g * 8, o);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    tc_fence_after();
    tmem_dealloc(tmem_base, tmem_cols);
  }
}

}  // namespace sb

using namespace sb;

// pooled runs: a window to be before, blocks to lie in, nothing that is defined by the distance of a key
static bool pool_valid(const WinParams& p) {
  return p.pool <= 0 || (p.window > 0 && p.pool_table && p.pool_blocks > 0 && p.kv_mode == kPaged && p.keep_first == 0 && !p.rel && !(p.bias_exp > 0.f) &&
                         !(p.softcap > 0.f));
}

static int win_grid(long long total) {
  long long b = (total + 255) / 256;
  const long long cap = (long long)num_sms() * 8;
  return (int)(b < 1 ? 1 : (b > cap ? cap : b));
}

extern "C" int sb_kv_append_split(const void* params, int f32, cudaStream_t stream) {
  const WinParams& p = *reinterpret_cast<const WinParams*>(params);
  if (p.T == 0) return 0;
  const int V = f32 ? 4 : 8;
  const bool vec = p.dk % V == 0 && p.dv % V == 0 && p.row_stride % V == 0 && p.k_off % V == 0 && p.v_off % V == 0;
  const int grid = win_grid((long long)p.T * p.Hkv * (p.dk + p.dv) / (vec ? V : 1));
  if (f32) {
    if (vec) kv_append_split_kernel<float, 4><<<grid, 256, 0, stream>>>(p);
    else kv_append_split_kernel<float, 1><<<grid, 256, 0, stream>>>(p);
  } else {
    if (vec) kv_append_split_kernel<__nv_bfloat16, 8><<<grid, 256, 0, stream>>>(p);
    else kv_append_split_kernel<__nv_bfloat16, 1><<<grid, 256, 0, stream>>>(p);
  }
  return (int)cudaGetLastError();
}

extern "C" int sb_attn_window_simt(const void* params, int f32, cudaStream_t stream) {
  const WinParams& p = *reinterpret_cast<const WinParams*>(params);
  if (p.T == 0) return 0;
  if (p.Hq % p.Hkv || p.Hq > 65535 || p.kv_mode == kPackedRows || (p.rel && p.rel_n < 1) || p.gate || (p.kv_mode == kLatent && p.dk != p.dv) || !pool_valid(p)) return -3;
  const size_t smem = (size_t)(p.dk + kSimtThreads + p.dv) * 4;
  if (smem > 48 * 1024) return -3;
  const dim3 grid(p.T, p.Hq);
  if (f32) window_simt_kernel<float><<<grid, kSimtThreads, smem, stream>>>(p);
  else window_simt_kernel<__nv_bfloat16><<<grid, kSimtThreads, smem, stream>>>(p);
  return (int)cudaGetLastError();
}

// Query tiles: rows tile_row[i] .. + tile_rows[i] - 1 (at most 128) of the packed buffer at positions tile_pos[i] .. of
// the sequence in cache slot tile_slot[i].
extern "C" int sb_attn_window_prefill(const void* params, const int* tile_row, const int* tile_rows, const int* tile_pos,
                                      const int* tile_slot, int n_tiles, int* status, cudaStream_t stream) {
  const WinParams& p = *reinterpret_cast<const WinParams*>(params);
  if (n_tiles == 0) return 0;
  if (p.Hq % p.Hkv || p.dk % 8 || p.dv % 8 || p.dk > 256 || p.dv > 256 || p.dk < 8 || p.dv < 8 || p.row_stride % 8 ||
      p.q_off % 8 || p.out_stride % 8 || p.out_off % 8 || p.block_elems % 8 || ((uintptr_t)p.out & 15) ||
      p.kv_mode == kLatent || p.gate_stride % 8 || ((uintptr_t)p.gate & 15) || (p.rel && (p.rel_n < 1 || p.bias_exp > 0.f)) || !pool_valid(p))
    return -2;
  static thread_local bool tl_context_bound = false;
  if (!tl_context_bound) {
    cudaFree(0);
    tl_context_bound = true;
  }
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x);
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.cache);
  CUtensorMap mq, mk, mv;
  // q: columns of one head x heads x rows, so that columns past dk read as zeros
  int r = make_tensor_map_bf16_3d(&mq, x + p.q_off, p.dk, p.Hq, p.T, p.dk, p.row_stride, 64, 1, 128);
  if (r) return r;
  if (p.kv_mode == kPackedRows) {
    // columns of one head x heads x key rows
    r = make_tensor_map_bf16_3d(&mk, cache, p.dk, p.Hkv, p.num_blocks, p.dk, p.block_elems, 64, 1, kWBlk);
    if (r) return r;
    r = make_tensor_map_bf16_3d(&mv, cache + (size_t)p.Hkv * p.dk, p.dv, p.Hkv, p.num_blocks, p.dv, p.block_elems, 64, 1,
                                kWBlk);
    if (r) return r;
  } else {
    r = make_tensor_map_bf16_3d(&mk, cache, p.dk, (long long)p.Hkv * kWBlk, p.num_blocks, p.dk, p.block_elems, 64, kWBlk, 1);
    if (r) return r;
    r = make_tensor_map_bf16_3d(&mv, cache + (size_t)p.Hkv * kWBlk * p.dk, p.dv, (long long)p.Hkv * kWBlk, p.num_blocks,
                                p.dv, p.block_elems, 64, kWBlk, 1);
    if (r) return r;
  }
  const WinSmem L((p.dk + 63) / 64, (p.dv + 63) / 64);
  const bool table = p.softcap > 0.f || p.rel;
  auto kernel = table ? window_prefill_kernel<true> : window_prefill_kernel<false>;
  static int configured[2] = {0, 0};
  if (configured[table] < L.total) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total);
    if (e != cudaSuccess) return (int)e;
    configured[table] = L.total;
  }
  const int need = 128 + (p.dv + 31) / 32 * 32;
  uint32_t cols = 256;
  while ((int)cols < need) cols *= 2;
  kernel<<<dim3(n_tiles, p.Hq), 160, L.total, stream>>>(mq, mk, mv, p, tile_row, tile_rows, tile_pos, tile_slot, cols,
                                                        status);
  return (int)cudaGetLastError();
}
