// Attention of single rows against a paged cache of latents (latent_params.h): every head's absorbed query meets the same
// R-wide rows, which are keys and values at once.  Also the cache append (norm fused) and the gather of cached rows.
//
// latent_decode_kernel (bf16, R a multiple of 8 up to 512).  The 64-token cache blocks ("tiles") of all rows form one list,
// (row, head group, tile), and every CTA of a persistent grid of one CTA per SM takes an equal range of it, whatever the
// context lengths.  A range is a few pieces, each a run of tiles of one (row, group); a piece that is not the whole
// sequence leaves a normalised partial result and its log-sum-exp in a workspace, two slots per CTA, and a small kernel
// merges them.  Six warps:
//   warp 4   producer: TMA ring of tiles, each [R / 64][64 tokens][64 columns], fetched once and used twice
//   warp 5   MMA issuer: S[head, token] = Qa C^T (128 x 64, rows past the group's heads are never read) one tile ahead of
//            O^T[column, head] += C^T P^T, where C^T is the A operand through an MN-major descriptor: the R columns fill
//            the 128 rows of the MMA whatever the number of heads, and O^T takes R / 128 * heads TMEM columns
//   warps 0..3   soft-max of the rows (heads) 32 w ..; together they rescale O^T (rarely: the reference maximum is only
//            raised when it grows by 2^8) and write the results
#include "common.cuh"
#include "launchers.h"
#include "latent_params.h"
#include "typed.cuh"

namespace sb {

constexpr int kLBlk = 64;
constexpr int kLMaxRows = 1024;     // rows (sequences) of one launch
constexpr int kLMaxHeads = 64;      // heads of a group
constexpr int kLMaxRank = 512;
constexpr int kLSmemLimit = 227 * 1024;

// ---------------------------------------------------------------------------------------
// append and gather
// ---------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(128) latent_append_kernel(LatentParams p, T* __restrict__ rows) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float gain = p.gain ? to_float(*reinterpret_cast<const T*>(p.gain)) : 1.f;
  for (int t = blockIdx.x * 4 + warp; t < p.T; t += gridDim.x * 4) {
    const T* z = reinterpret_cast<const T*>(p.x) + (size_t)t * p.row_stride + p.c_off;
    float ss = 0.f;
    for (int c = lane * V; c < p.R; c += 32 * V) {
      float v[V];
      load_vec<T, V>(z + c, v);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(gain * v[i], gain * v[i], ss);
    }
    const float f = gain / sqrtf(warp_sum(ss) / (float)p.R + p.eps);
    const int slot = p.seq_ids[t], pos = p.positions[t];
    T* dst = nullptr;
    if (slot >= 0 && pos >= 0 && pos / kLBlk < p.max_blocks) {
      const int blk = p.block_table[(size_t)slot * p.max_blocks + pos / kLBlk];
      if (blk >= 0 && blk < p.num_blocks) dst = reinterpret_cast<T*>(p.cache) + ((size_t)blk * kLBlk + pos % kLBlk) * p.R;
    }
    if (!dst && !rows) continue;
    for (int c = lane * V; c < p.R; c += 32 * V) {
      float v[V], w[V];
      load_vec<T, V>(z + c, v);
      load_vec<T, V>(reinterpret_cast<const T*>(p.c_norm) + c, w);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] *= f * w[i];
      if (dst) store_vec<T, V>(dst + c, v);
      if (rows) store_vec<T, V>(rows + (size_t)t * p.R + c, v);
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(128) latent_gather_kernel(LatentParams p, const int* __restrict__ key_slot,
                                                            const int* __restrict__ key_pos, T* __restrict__ rows, int n) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int t = blockIdx.x * 4 + warp; t < n; t += gridDim.x * 4) {
    const int slot = key_slot[t], pos = key_pos[t];
    const int blk = pos / kLBlk < p.max_blocks ? p.block_table[(size_t)slot * p.max_blocks + pos / kLBlk] : -1;
    const bool ok = blk >= 0 && blk < p.num_blocks;      // always, for positions a sequence holds
    const T* src = reinterpret_cast<const T*>(p.cache) + ((size_t)(ok ? blk : 0) * kLBlk + pos % kLBlk) * p.R;
    for (int c = lane * V; c < p.R; c += 32 * V) {
      float v[V];
      load_vec<T, V>(src + c, v);
      if (!ok)
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = 0.f;
      store_vec<T, V>(rows + (size_t)t * p.R + c, v);
    }
  }
}

// ---------------------------------------------------------------------------------------
// decode
// ---------------------------------------------------------------------------------------
struct LdLayout {
  int chunks, mchunks, hg, groups, stages, stage_bytes;
  int kv_off, p_off, pre_off, stat_off, bar_off, total;
  __host__ __device__ LdLayout(int H, int R, int T) {
    chunks = (R + 63) / 64;
    mchunks = (R + 127) / 128;
    groups = (H + kLMaxHeads - 1) / kLMaxHeads;
    hg = ((H + groups - 1) / groups + 15) / 16 * 16;       // heads of a group: a legal N of the O^T MMA
    stage_bytes = chunks * 8192;
    kv_off = chunks * hg * 128;
    const int p_bytes = hg * 128;
    const int fixed = kv_off + 2 * p_bytes + (T + 1) * 4 + 2048;
    stages = (kLSmemLimit - fixed) / stage_bytes;
    if (stages > 8) stages = 8;
    p_off = kv_off + stages * stage_bytes;
    stat_off = p_off + 2 * p_bytes;                        // alpha [2][64], l [64], m [64], need [2][4]
    bar_off = stat_off + (4 * kLMaxHeads + 8) * 4;
    pre_off = bar_off + (2 * stages + 12) * 8 + 16;
    total = pre_off + (T + 1) * 4;
    const int least = p_off + 8192;                        // the over-read of the last stage stays inside
    if (total < least) total = least;
    if (total < kv_off + 16384) total = kv_off + 16384;    // ... and that of the last query chunk
  }
};

struct LdParams {
  const int* seq_ids;
  const int* positions;
  const int* block_table;
  long long num_blocks;
  int max_blocks, T, H, R;
  float scale_log2;
  const __nv_bfloat16* gain;
  __nv_bfloat16* out;       // [T, H, R]
  float* ws_o;              // [2 * grid][hg][R]
  float* ws_lse;            // [2 * grid][hg]
  int* ws_pre;              // [T + 1] tiles before each row, written by the first CTA
  int* status;
};

__device__ __forceinline__ int ld_tiles(const LdParams& p, int t) {
  const int pos = p.seq_ids[t] >= 0 ? p.positions[t] : -1;
  return pos < 0 ? 0 : min(pos / kLBlk + 1, p.max_blocks);
}

__device__ __forceinline__ int ld_range(long long total, int cta, int grid) { return (int)(total * cta / grid); }

struct LdPiece {
  int row, group, t0, n, tiles;
  bool whole;
};

// the piece at list position `cur` of a range that ends at `end`; pre[t] = tiles of rows before t
__device__ __forceinline__ LdPiece ld_piece(const int* pre, int T, int groups, int cur, int end) {
  int lo = 0, hi = T;       // the last row that begins at or before cur (rows without tiles have no width)
  while (hi - lo > 1) {
    const int mid = (lo + hi) / 2;
    if (pre[mid] * groups <= cur) lo = mid;
    else hi = mid;
  }
  LdPiece q;
  q.row = lo;
  q.tiles = pre[lo + 1] - pre[lo];
  const int at = cur - pre[lo] * groups;
  q.group = at / q.tiles;
  q.t0 = at - q.group * q.tiles;
  q.n = min(q.tiles - q.t0, end - cur);
  q.whole = q.n == q.tiles;
  return q;
}

__global__ void __launch_bounds__(192, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap map_c, const __grid_constant__ CUtensorMap map_q, LdParams p) {
  const LdLayout L(p.H, p.R, p.T);
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw;
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, (int)kStatusBadArgument);
    return;
  }
  uint8_t* sQ = smem;
  uint8_t* sC = smem + L.kv_off;
  uint8_t* sP = smem + L.p_off;
  float* s_alpha = reinterpret_cast<float*>(smem + L.stat_off);       // [2][64]
  float* s_l = s_alpha + 2 * kLMaxHeads;
  float* s_m = s_l + kLMaxHeads;
  int* s_need = reinterpret_cast<int*>(s_m + kLMaxHeads);             // [2][4]
  uint64_t* c_full = reinterpret_cast<uint64_t*>(smem + L.bar_off);
  uint64_t* c_empty = c_full + L.stages;
  uint64_t* q_full = c_empty + L.stages;
  uint64_t* q_empty = q_full + 1;
  uint64_t* s_full = q_empty + 1;       // [2]
  uint64_t* s_empty = s_full + 2;       // [2]
  uint64_t* p_full = s_empty + 2;       // [2]
  uint64_t* p_empty = p_full + 2;       // [2]: the MMAs that read P have completed
  uint64_t* o_full = p_empty + 2;
  uint64_t* o_empty = o_full + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_empty + 1);
  int* s_pre = reinterpret_cast<int*>(smem + L.pre_off);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int heads_per_group = (p.H + L.groups - 1) / L.groups;
  const int soft_warps = (heads_per_group + 31) / 32;                 // warps with heads of their own
  constexpr uint32_t kTmemCols = 512;                                 // S: 2 x 64, O^T: mchunks x hg columns

  if (tid == 0) {
    tma_prefetch_desc(&map_c);
    tma_prefetch_desc(&map_q);
    for (int i = 0; i < 2 * L.stages + 2; ++i) mbar_init(&c_full[i], 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], soft_warps);
      mbar_init(&p_full[i], 4);
      mbar_init(&p_empty[i], 1);
    }
    mbar_init(o_full, 1);
    mbar_init(o_empty, 4);
    fence_barrier_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  if (warp == 4) {
    // running sum of the rows' tiles
    int base = 0;
    for (int t0 = 0; t0 < p.T; t0 += 32) {
      const int t = t0 + lane;
      int v = t < p.T ? ld_tiles(p, t) : 0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += u;
      }
      if (t < p.T) s_pre[t + 1] = base + v;
      base += __shfl_sync(0xffffffffu, v, 31);
    }
    if (lane == 0) s_pre[0] = 0;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 128;
  const long long total = (long long)s_pre[p.T] * L.groups;
  const int begin = ld_range(total, blockIdx.x, gridDim.x), end = ld_range(total, blockIdx.x + 1, gridDim.x);
  if (blockIdx.x == 0)
    for (int i = tid; i <= p.T; i += blockDim.x) p.ws_pre[i] = s_pre[i];

  if (warp == 4) {
    // ------------------------------ producer ------------------------------
    if (lane == 0) {
      uint32_t tile_no = 0, piece_no = 0;
      bool ok = true;
      for (int cur = begin; cur < end && ok;) {
        const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
        const int* blocks = p.block_table + (size_t)p.seq_ids[q.row] * p.max_blocks;
        for (int t = 0; t < q.n && ok; ++t, ++tile_no) {
          const int stage = tile_no % L.stages;
          if (!mbar_wait(&c_empty[stage], ((tile_no / L.stages) & 1) ^ 1, p.status, kStatusTimeoutProducer)) {
            ok = false;
            break;
          }
          int blk = blocks[q.t0 + t];
          if (blk < 0 || blk >= p.num_blocks) blk = 0;      // never among the visible blocks of a well-formed table
          uint8_t* dst = sC + stage * L.stage_bytes;
          mbar_arrive_expect_tx(&c_full[stage], (uint32_t)L.stage_bytes);
          for (int c = 0; c < L.chunks; ++c) tma_load_3d(dst + c * 8192, &map_c, &c_full[stage], c * 64, 0, blk);
          if (t == 0) {     // after the piece's first tile: the queries wait for the score MMAs of the piece before
            if (!mbar_wait(q_empty, (piece_no & 1) ^ 1, p.status, kStatusTimeoutProducer)) {
              ok = false;
              ++tile_no;
              break;
            }
            mbar_arrive_expect_tx(q_full, (uint32_t)(L.chunks * L.hg * 128));
            for (int c = 0; c < L.chunks; ++c)
              tma_load_3d(sQ + c * L.hg * 128, &map_q, q_full, c * 64, q.group * heads_per_group, q.row);
          }
        }
        ++piece_no;
        cur += q.n;
      }
      if (!ok) {      // no copy may be in flight when shared memory is given back
        const uint32_t first = tile_no > (uint32_t)L.stages ? tile_no - L.stages : 0;
        for (uint32_t j = first; j < tile_no; ++j) mbar_wait(&c_full[j % L.stages], (j / L.stages) & 1, nullptr, 0);
      }
    }
  } else if (warp == 5) {
    // ------------------------------ MMA issuer ------------------------------
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(128, kLBlk, 0, 0);
      const uint32_t idesc_o = umma_idesc_bf16(128, L.hg, 1, 0);
      const int k_steps = (p.R + 15) / 16;
      const uint32_t aq = smem_u32(sQ);
      uint32_t first = 0, piece_no = 0;
      bool ok = true;
      for (int cur = begin; cur < end && ok; ++piece_no) {
        const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
        if (!mbar_wait(q_full, piece_no & 1, p.status, kStatusTimeoutMma)) break;
        for (int t = 0; t <= q.n && ok; ++t) {
          if (t < q.n) {
            const uint32_t tn = first + t;
            const int stage = tn % L.stages, sb_ = tn & 1;
            if (!mbar_wait(&c_full[stage], (tn / L.stages) & 1, p.status, kStatusTimeoutMma) ||
                !mbar_wait(&s_empty[sb_], ((tn >> 1) & 1) ^ 1, p.status, kStatusTimeoutMma)) {
              ok = false;
              break;
            }
            tc_fence_after();
            const uint32_t bc = smem_u32(sC + stage * L.stage_bytes);
            for (int kk = 0; kk < k_steps; ++kk) {
              const uint64_t da = umma_smem_desc(aq + (kk / 4) * (L.hg * 128) + (kk % 4) * 32, 16, 1024);
              const uint64_t db = umma_smem_desc(bc + (kk / 4) * 8192 + (kk % 4) * 32, 16, 1024);
              umma_bf16_ss(tmem_s + sb_ * 64, da, db, idesc_s, kk ? 1u : 0u);
            }
            umma_commit(&s_full[sb_]);
            if (t == q.n - 1) umma_commit(q_empty);
          }
          if (t > 0) {
            const uint32_t tn = first + t - 1;
            const int stage = tn % L.stages, pb = tn & 1;
            if (!mbar_wait(&p_full[pb], (tn >> 1) & 1, p.status, kStatusTimeoutMma) ||
                (t == 1 && !mbar_wait(o_empty, (piece_no & 1) ^ 1, p.status, kStatusTimeoutMma))) {
              ok = false;
              break;
            }
            tc_fence_after();
            const uint32_t ac = smem_u32(sC + stage * L.stage_bytes), bp = smem_u32(sP + pb * L.hg * 128);
            for (int mc = 0; mc < L.mchunks; ++mc)
#pragma unroll
              for (int kk = 0; kk < kLBlk / 16; ++kk) {
                const uint64_t da = umma_smem_desc(ac + mc * 16384 + kk * 2048, 8192, 1024);
                const uint64_t db = umma_smem_desc(bp + kk * 32, 16, 1024);
                umma_bf16_ss(tmem_o + mc * L.hg, da, db, idesc_o, (t > 1 || kk) ? 1u : 0u);
              }
            umma_commit(&c_empty[stage]);
            umma_commit(&p_empty[pb]);
            if (t == q.n) umma_commit(o_full);
          }
        }
        first += q.n;
        cur += q.n;
      }
    }
  } else {
    // ------------------------------ soft-max, rescaling and output (warps 0..3) ------------------------------
    const float gain = p.gain ? __bfloat162float(*p.gain) : 1.f;
    const float scale_log2 = p.scale_log2 * gain;
    const uint32_t lane_off = (uint32_t)(warp * 32) << 16;
    const int row_head = warp * 32 + lane;          // head of the group whose scores this thread holds
    const bool soft = warp < soft_warps;
    uint32_t first = 0, piece_no = 0;
    // the four warps meet at a named barrier in every tile and leave the loop together when a wait of one ran out
    bool mine = true;
    auto meet = [&]() -> bool { return !named_barrier_or(1, 128, !mine); };
    bool ok = true;
    for (int cur = begin; cur < end && ok; ++piece_no) {
      const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
      const int ctx = p.positions[q.row] + 1;
      const int head0 = q.group * heads_per_group;
      const int nh = min(heads_per_group, p.H - head0);
      float m_ref = 0.f, l_run = 0.f;
      for (int t = 0; t < q.n && ok; ++t) {
        const uint32_t tn = first + t;
        const int sb_ = tn & 1;
        float sv[kLBlk];
        float m_tile = -INFINITY;
        bool need = false;
        if (soft && mine) {
          mine = __all_sync(0xffffffffu, mbar_wait(&s_full[sb_], (tn >> 1) & 1, p.status, kStatusTimeoutEpilogue));
          if (mine) {
            tc_fence_after();
            uint32_t r0[32], r1[32];
            tmem_ld_32x32(tmem_s + lane_off + sb_ * 64, r0);
            tmem_ld_32x32(tmem_s + lane_off + sb_ * 64 + 32, r1);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_empty[sb_]);
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              sv[i] = __uint_as_float(r0[i]) * scale_log2;
              sv[32 + i] = __uint_as_float(r1[i]) * scale_log2;
            }
            const int kv0 = (q.t0 + t) * kLBlk;
            if (kv0 + kLBlk > ctx) {
#pragma unroll
              for (int i = 0; i < kLBlk; ++i)
                if (kv0 + i >= ctx) sv[i] = -INFINITY;
            }
#pragma unroll
            for (int i = 0; i < kLBlk; ++i) m_tile = fmaxf(m_tile, sv[i]);
            if (t == 0) m_ref = m_tile;             // a tile of a row holds at least one visible key
            else need = __any_sync(0xffffffffu, row_head < nh && m_tile > m_ref + 8.f);
          }
        }
        if (t > 0) {
          if (soft) {
            float alpha = 1.f;
            if (need) {
              const float m_new = fmaxf(m_ref, m_tile);
              alpha = exp2f(m_ref - m_new);
              m_ref = m_new;
              l_run *= alpha;
            }
            s_alpha[(t & 1) * kLMaxHeads + row_head] = alpha;
          }
          if (lane == 0) s_need[(t & 1) * 4 + warp] = need ? 1 : 0;
        }
        ok = meet();
        if (!ok) break;
        if (t > 0 && (s_need[(t & 1) * 4] | s_need[(t & 1) * 4 + 1])) {
          // raise the reference maximum: O^T column h times alpha[h], once PV(t - 1) has completed
          const uint32_t tp = tn - 1;
          if (!__all_sync(0xffffffffu, mbar_wait(&p_empty[tp & 1], (tp >> 1) & 1, p.status, kStatusTimeoutEpilogue))) {
            mine = false;
          } else {
            tc_fence_after();
            const float* al = s_alpha + (t & 1) * kLMaxHeads;
#pragma unroll 1
            for (int mc = 0; mc < L.mchunks; ++mc)
#pragma unroll 1
              for (int c = 0; c < L.hg; c += 16) {
                uint32_t r[16];
                tmem_ld_32x16(tmem_o + lane_off + mc * L.hg + c, r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * al[c + i]);
                tmem_st_32x16(tmem_o + lane_off + mc * L.hg + c, r);
              }
            tmem_st_wait();
          }
        }
        if (mine) mine = __all_sync(0xffffffffu, mbar_wait(&p_empty[sb_], ((tn >> 1) & 1) ^ 1, p.status, kStatusTimeoutEpilogue));
        if (soft && mine) {
          uint32_t pk[kLBlk / 2];
          float rsum = 0.f;
#pragma unroll
          for (int i = 0; i < kLBlk; i += 2) {
            const float p0 = exp2f(sv[i] - m_ref), p1 = exp2f(sv[i + 1] - m_ref);
            rsum += p0 + p1;
            pk[i / 2] = pack_bf16x2(p0, p1);
          }
          l_run += rsum;
          if (row_head < L.hg) {
            uint8_t* prow = sP + sb_ * L.hg * 128 + row_head * 128;
#pragma unroll
            for (int piece = 0; piece < 8; ++piece) {
              uint4 v = make_uint4(pk[piece * 4], pk[piece * 4 + 1], pk[piece * 4 + 2], pk[piece * 4 + 3]);
              if (row_head >= nh) v = make_uint4(0, 0, 0, 0);
              *reinterpret_cast<uint4*>(prow + ((piece ^ (row_head & 7)) << 4)) = v;
            }
          }
          fence_proxy_async_smem();
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[sb_]);
      }
      if (!ok) break;
      if (soft) {
        s_l[row_head] = l_run;
        s_m[row_head] = m_ref;
      }
      mine = mine && __all_sync(0xffffffffu, mbar_wait(o_full, piece_no & 1, p.status, kStatusTimeoutEpilogue));
      ok = meet();
      if (!ok) break;
      tc_fence_after();
      const int slot = 2 * blockIdx.x + (cur == begin ? 0 : 1);
      __nv_bfloat16* orow = p.out + ((size_t)q.row * p.H + head0) * p.R;
      float* wrow = p.ws_o + (size_t)slot * L.hg * p.R;
#pragma unroll 1
      for (int mc = 0; mc < L.mchunks; ++mc) {
        const int col = mc * 128 + warp * 32 + lane;
#pragma unroll 1
        for (int c = 0; c < nh; c += 16) {
          uint32_t r[16];
          tmem_ld_32x16(tmem_o + lane_off + mc * L.hg + c, r);
          tmem_ld_wait();
          if (col < p.R) {
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              if (c + i >= nh) break;
              const float v = __uint_as_float(r[i]) / s_l[c + i];      // the sum is at least one: a row's maximum has weight one
              if (q.whole) orow[(size_t)(c + i) * p.R + col] = __float2bfloat16(v);
              else wrow[(size_t)(c + i) * p.R + col] = v;
            }
          }
        }
      }
      if (!q.whole && warp == 0)
        for (int h = lane; h < nh; h += 32) p.ws_lse[(size_t)slot * L.hg + h] = s_m[h] + log2f(s_l[h]);
      tc_fence_before();
      ok = meet();      // statistics and O^T have been read
      if (lane == 0) mbar_arrive(o_empty);
      first += q.n;
      cur += q.n;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

// rows whose tiles are spread over several CTAs: weighted mean of the partial results; zero rows for idle slots
__global__ void __launch_bounds__(128) latent_merge_kernel(LdParams p, int hg, int groups, int grid) {
  const int row = blockIdx.x, h = blockIdx.y, group = h / ((p.H + groups - 1) / groups);
  const int hl = h - group * ((p.H + groups - 1) / groups);
  const int tiles = p.ws_pre[row + 1] - p.ws_pre[row];
  __nv_bfloat16* orow = p.out + ((size_t)row * p.H + h) * p.R;
  if (tiles == 0) {
    for (int d = threadIdx.x; d < p.R; d += blockDim.x) orow[d] = __float2bfloat16(0.f);
    return;
  }
  const long long total = (long long)p.ws_pre[p.T] * groups;
  const long long s0 = (long long)p.ws_pre[row] * groups + (long long)group * tiles, s1 = s0 + tiles - 1;
  const int c0 = (int)(((s0 + 1) * grid - 1) / total), c1 = (int)(((s1 + 1) * grid - 1) / total);
  if (c0 == c1) return;
  auto slot_of = [&](int c) { return 2 * c + (c == c0 && ld_range(total, c, grid) != s0 ? 1 : 0); };
  float m = -INFINITY;
  for (int c = c0; c <= c1; ++c)
    if (ld_range(total, c, grid) != ld_range(total, c + 1, grid)) m = fmaxf(m, p.ws_lse[(size_t)slot_of(c) * hg + hl]);
  for (int d = threadIdx.x; d < p.R; d += blockDim.x) {
    float acc = 0.f, wsum = 0.f;
    for (int c = c0; c <= c1; ++c) {
      if (ld_range(total, c, grid) == ld_range(total, c + 1, grid)) continue;      // a CTA without tiles
      const size_t at = (size_t)slot_of(c) * hg + hl;
      const float w = exp2f(p.ws_lse[at] - m);
      wsum += w;
      acc += w * p.ws_o[at * p.R + d];
    }
    orow[d] = __float2bfloat16(acc / wsum);
  }
}

}  // namespace sb

using namespace sb;

// rows (may be null): a copy of the appended rows, [T, R]
extern "C" int sb_latent_append(const void* params, void* rows, int f32, cudaStream_t stream) {
  const LatentParams& p = *reinterpret_cast<const LatentParams*>(params);
  if (p.T <= 0) return 0;
  const int V = f32 ? 4 : 8;
  const bool vec = p.R % V == 0 && p.c_off % V == 0 && p.row_stride % V == 0;
  const int blocks = (p.T + 3) / 4, cap = num_sms() * 16, grid = blocks < cap ? blocks : cap;
  using B = __nv_bfloat16;
  if (f32) {
    if (vec) latent_append_kernel<float, 4><<<grid, 128, 0, stream>>>(p, (float*)rows);
    else latent_append_kernel<float, 1><<<grid, 128, 0, stream>>>(p, (float*)rows);
  } else {
    if (vec) latent_append_kernel<B, 8><<<grid, 128, 0, stream>>>(p, (B*)rows);
    else latent_append_kernel<B, 1><<<grid, 128, 0, stream>>>(p, (B*)rows);
  }
  return (int)cudaGetLastError();
}

// rows [n, R]: the cached latents of (key_slot[i], key_pos[i])
extern "C" int sb_latent_gather(const void* params, const int* key_slot, const int* key_pos, void* rows, int n, int f32,
                                cudaStream_t stream) {
  const LatentParams& p = *reinterpret_cast<const LatentParams*>(params);
  if (n <= 0) return 0;
  const int V = f32 ? 4 : 8;
  const int blocks = (n + 3) / 4, cap = num_sms() * 16, grid = blocks < cap ? blocks : cap;
  using B = __nv_bfloat16;
  if (f32) {
    if (p.R % V == 0) latent_gather_kernel<float, 4><<<grid, 128, 0, stream>>>(p, key_slot, key_pos, (float*)rows, n);
    else latent_gather_kernel<float, 1><<<grid, 128, 0, stream>>>(p, key_slot, key_pos, (float*)rows, n);
  } else {
    if (p.R % V == 0) latent_gather_kernel<B, 8><<<grid, 128, 0, stream>>>(p, key_slot, key_pos, (B*)rows, n);
    else latent_gather_kernel<B, 1><<<grid, 128, 0, stream>>>(p, key_slot, key_pos, (B*)rows, n);
  }
  return (int)cudaGetLastError();
}

// head groups of the tensor-core kernel, or 0 when the sizes need the general one
extern "C" int sb_latent_decode_groups(int H, int R) {
  if (H < 1 || R < 8 || R % 8 || R > kLMaxRank) return 0;
  const LdLayout L(H, R, kLMaxRows);
  return L.stages >= 2 && 128 + L.mchunks * L.hg <= 512 ? L.groups : 0;
}

extern "C" int sb_latent_decode_grid() { return num_sms(); }

// Row t (cache slot seq_ids[t], at most 1024 rows) attends to positions 0 .. positions[t]; seq_ids[t] < 0: its result is
// zero.  Workspaces: ws_o 2 * grid * heads of a group (rounded up to 16) * R floats, ws_stat 2 * grid * heads + 1025 words.
extern "C" int sb_latent_decode(const void* params, float* ws_o, float* ws_stat, int* status, cudaStream_t stream) {
  const LatentParams& w = *reinterpret_cast<const LatentParams*>(params);
  if (w.T <= 0) return 0;
  const int groups = sb_latent_decode_groups(w.H, w.R);
  if (!groups || w.T > kLMaxRows || ((uintptr_t)w.qa & 15) || ((uintptr_t)w.cache & 15)) return -2;
  static thread_local bool tl_context_bound = false;
  if (!tl_context_bound) {
    cudaFree(0);
    tl_context_bound = true;
  }
  const LdLayout L(w.H, w.R, w.T);
  CUtensorMap mc, mq;
  int r = make_tensor_map_bf16_3d(&mc, w.cache, w.R, kLBlk, w.num_blocks, w.R, (long long)kLBlk * w.R, 64, kLBlk, 1);
  if (r) return r;
  r = make_tensor_map_bf16_3d(&mq, w.qa, w.R, w.H, w.T, w.R, (long long)w.H * w.R, 64, L.hg, 1);
  if (r) return r;
  const int grid = num_sms();
  LdParams p;
  p.seq_ids = w.seq_ids; p.positions = w.positions; p.block_table = w.block_table; p.num_blocks = w.num_blocks;
  p.max_blocks = w.max_blocks; p.T = w.T; p.H = w.H; p.R = w.R;
  p.scale_log2 = w.scale * 1.4426950408889634f;
  p.gain = reinterpret_cast<const __nv_bfloat16*>(w.gain);
  p.out = reinterpret_cast<__nv_bfloat16*>(w.out);
  p.ws_o = ws_o; p.ws_lse = ws_stat; p.ws_pre = reinterpret_cast<int*>(ws_stat + (size_t)2 * grid * L.hg);
  p.status = status;
  static int configured = 0;
  if (configured < L.total) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total);
    if (e != cudaSuccess) return (int)e;
    configured = L.total;
  }
  latent_decode_kernel<<<grid, 192, L.total, stream>>>(mc, mq, p);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  latent_merge_kernel<<<dim3(w.T, w.H), 128, 0, stream>>>(p, L.hg, L.groups, grid);
  return (int)cudaGetLastError();
}
