// Attention of single rows against a paged cache of latents (latent_params.h): every head's absorbed query meets the same
// R-wide rows, which are keys and values at once.  Also the cache append (norm fused) and the gather of cached rows.
//
// latent_decode_kernel (bf16, R a multiple of 8 up to 512).  The 64-token cache blocks ("tiles") of all rows form one list,
// (row, group of at most 32 heads, tile), and every CTA of a persistent grid of one CTA per SM takes an equal range of it,
// whatever the context lengths.  A range is a few pieces, each a run of tiles of one (row, group); a piece that is not the
// whole sequence leaves a normalised partial result and its log-sum-exp in a workspace, two slots per CTA, and a small
// kernel merges them.  The warps:
//   5        producer: TMA ring of tiles, each [R / 64][64 tokens][64 columns], fetched once and used twice
//   8        queries of the piece -> TMEM (row = lane), the A operand of the score product: they cost no shared memory,
//            which leaves room for three tiles of 512 columns
//   6        MMA issuer: S[head, token] = Qa C^T (128 x 64, rows past the group's heads are never read) one tile ahead of
//            O^T[column, head] += C^T P^T, where C^T is the A operand through an MN-major descriptor: the R columns fill
//            the 128 rows of the MMA whatever the number of heads, and O^T takes R / 128 * heads TMEM columns
//   0        soft-max (thread = head); the reference maximum is only raised when it grows by 2^8
//   4, 1..3  rows 0..31, 32..127 of O^T: called by the soft-max warp to rescale it (rarely) and to write a piece's result
//            while the next piece's first tiles are under way
//   7        idle (TMEM rows belong to warps by their index modulo four)
#include "common.cuh"
#include "launchers.h"
#include "latent_params.h"
#include "typed.cuh"

namespace sb {

constexpr int kLBlk = 64;
constexpr int kLMaxRows = 1024;     // rows (sequences) of one launch
constexpr int kLMaxHeads = 32;      // heads of a group
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
  int p_off, stat_off, bar_off, pre_off, total;
  __host__ __device__ LdLayout(int H, int R, int T) {
    chunks = (R + 63) / 64;
    mchunks = (R + 127) / 128;
    groups = (H + kLMaxHeads - 1) / kLMaxHeads;
    hg = ((H + groups - 1) / groups + 15) / 16 * 16;       // heads of a group: a legal N of the O^T MMA
    stage_bytes = chunks * 8192;
    const int p_bytes = hg * 128;
    const int fixed = 2 * p_bytes + (T + 1) * 4 + 2048;
    stages = (kLSmemLimit - fixed) / stage_bytes;
    if (stages > 8) stages = 8;
    p_off = stages * stage_bytes;
    stat_off = p_off + 2 * p_bytes;                        // alpha [32], 1 / l [32], log-sum-exp [32], call [2]
    bar_off = stat_off + (3 * kLMaxHeads + 2) * 4;
    pre_off = bar_off + (2 * stages + 14) * 8 + 16;
    total = pre_off + (T + 1) * 4;
    if (total < p_off + 8192) total = p_off + 8192;        // an odd chunk count reads (and drops) one chunk past a stage
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
  const __nv_bfloat16* qa;  // [T, H, R]
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

__global__ void __launch_bounds__(288, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap map_c, LdParams p) {
  const LdLayout L(p.H, p.R, p.T);
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw;
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, (int)kStatusBadArgument);
    return;
  }
  uint8_t* sC = smem;
  uint8_t* sP = smem + L.p_off;
  float* s_alpha = reinterpret_cast<float*>(smem + L.stat_off);       // [32]
  float* s_l = s_alpha + kLMaxHeads;
  float* s_m = s_l + kLMaxHeads;
  int* s_call = reinterpret_cast<int*>(s_m + kLMaxHeads);             // 0: rescale, 1: the piece has ended
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
  uint64_t* call = o_empty + 1;         // soft-max warp -> O^T warps
  uint64_t* answer = call + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(answer + 1);
  int* s_pre = reinterpret_cast<int*>(smem + L.pre_off);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int heads_per_group = (p.H + L.groups - 1) / L.groups;
  constexpr uint32_t kTmemCols = 512;                                 // S: 2 x 64, O^T: mchunks * hg, Qa: chunks * 32

  if (tid == 0) {
    tma_prefetch_desc(&map_c);
    for (int i = 0; i < 2 * L.stages + 2; ++i) mbar_init(&c_full[i], 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 1);
      mbar_init(&p_full[i], 1);
      mbar_init(&p_empty[i], 1);
    }
    mbar_init(o_full, 1);
    mbar_init(o_empty, 4);
    mbar_init(call, 1);
    mbar_init(answer, 4);
    fence_barrier_init();
  }
  if (warp == 6) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  for (int t = tid; t < p.T; t += blockDim.x) s_pre[t + 1] = ld_tiles(p, t);
  __syncthreads();
  if (warp == 8) {
    // running sum of the rows' tiles
    int base = 0;
    for (int t0 = 0; t0 < p.T; t0 += 32) {
      const int t = t0 + lane;
      int v = t < p.T ? s_pre[t + 1] : 0;
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
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 128, tmem_q = tmem_base + 256;
  const long long total = (long long)s_pre[p.T] * L.groups;
  const int begin = ld_range(total, blockIdx.x, gridDim.x), end = ld_range(total, blockIdx.x + 1, gridDim.x);
  if (blockIdx.x == 0)
    for (int i = tid; i <= p.T; i += blockDim.x) p.ws_pre[i] = s_pre[i];

  if (warp == 5) {
    // ------------------------------ producer ------------------------------
    if (lane == 0) {
      uint32_t tile_no = 0;
      bool ok = true;
      for (int cur = begin; cur < end && ok;) {
        const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
        const int* blocks = p.block_table + (size_t)p.seq_ids[q.row] * p.max_blocks + q.t0;
        int next = blocks[0];
        for (int t = 0; t < q.n; ++t, ++tile_no) {
          int blk = next;
          if (t + 1 < q.n) next = blocks[t + 1];            // read before the wait
          if (blk < 0 || blk >= p.num_blocks) blk = 0;      // never among the visible blocks of a well-formed table
          const int stage = tile_no % L.stages;
          if (!mbar_wait(&c_empty[stage], ((tile_no / L.stages) & 1) ^ 1, p.status, kStatusTimeoutProducer)) {
            ok = false;
            break;
          }
          uint8_t* dst = sC + stage * L.stage_bytes;
          mbar_arrive_expect_tx(&c_full[stage], (uint32_t)L.stage_bytes);
          for (int c = 0; c < L.chunks; ++c) tma_load_3d(dst + c * 8192, &map_c, &c_full[stage], c * 64, 0, blk);
        }
        cur += q.n;
      }
      if (!ok) {      // no copy may be in flight when shared memory is given back
        const uint32_t first = tile_no > (uint32_t)L.stages ? tile_no - L.stages : 0;
        for (uint32_t j = first; j < tile_no; ++j) mbar_wait(&c_full[j % L.stages], (j / L.stages) & 1, nullptr, 0);
      }
    }
  } else if (warp == 8) {
    // ------------------------------ queries -> TMEM (lane = head) ------------------------------
    uint32_t piece_no = 0;
    for (int cur = begin; cur < end; ++piece_no) {
      const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
      const int head0 = q.group * heads_per_group;
      const bool mine = head0 + lane < p.H && lane < heads_per_group;
      const __nv_bfloat16* src = p.qa + ((size_t)q.row * p.H + head0 + (mine ? lane : 0)) * p.R;
      if (mine)
        for (int c = 0; c < p.R; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(src + c));
      // the score MMAs of the piece before have read theirs
      if (!__all_sync(0xffffffffu, mbar_wait(q_empty, (piece_no & 1) ^ 1, p.status, kStatusTimeoutProducer))) break;
      tc_fence_after();
#pragma unroll 2
      for (int c = 0; c < L.chunks; ++c) {
        uint32_t r[32];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          uint4 v = make_uint4(0, 0, 0, 0);
          if (mine && c * 64 + i * 8 < p.R) v = *reinterpret_cast<const uint4*>(src + c * 64 + i * 8);
          r[4 * i] = v.x; r[4 * i + 1] = v.y; r[4 * i + 2] = v.z; r[4 * i + 3] = v.w;
        }
        tmem_st_32x32(tmem_q + c * 32, r);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(q_full);
      cur += q.n;
    }
  } else if (warp == 6) {
    // ------------------------------ MMA issuer (the whole warp, converged; one lane issues) ------------------------------
    const uint32_t leader = elect_one() ? 1u : 0u;
    const uint32_t idesc_s = umma_idesc_bf16(128, kLBlk, 0, 0);
    const uint32_t idesc_o = umma_idesc_bf16(128, L.hg, 1, 0);
    // descriptors differ in their address field (16-byte units) only.  Columns past R are zeros in both operands of S.
    const uint64_t dc = umma_smem_desc(smem_u32(sC), 16, 1024);
    const uint64_t dt = umma_smem_desc(smem_u32(sC), 8192, 1024), dp = umma_smem_desc(smem_u32(sP), 16, 1024);
    const uint32_t p_buf = L.hg * 8, stage_step = L.stage_bytes >> 4;
    const int stages = L.stages;
    // ring positions and phases of the tile whose scores / whose weighted sum comes next
    int s_stage = 0, o_stage = 0;
    uint32_t s_phase = 0, s_tile = 0, o_tile = 0, piece_no = 0;
    bool ok = true;
    for (int cur = begin; cur < end && ok; ++piece_no) {
      const int n = __shfl_sync(0xffffffffu, ld_piece(s_pre, p.T, L.groups, cur, end).n, 0);
      if (!mbar_wait(q_full, piece_no & 1, p.status, kStatusTimeoutMma)) break;
      for (int t = 0; t <= n && ok; ++t) {
        if (t < n) {
          const uint32_t sb_ = s_tile & 1;
          if (!mbar_wait(&c_full[s_stage], s_phase, p.status, kStatusTimeoutMma) ||
              !mbar_wait(&s_empty[sb_], ((s_tile >> 1) & 1) ^ 1, p.status, kStatusTimeoutMma)) {
            ok = false;
            break;
          }
          tc_fence_after();
          const uint32_t d = tmem_s + sb_ * 64;
          uint64_t db = dc + (uint32_t)s_stage * stage_step;
          uint32_t a = tmem_q;
#pragma unroll 1
          for (int c = 0; c < L.chunks; ++c, a += 32, db += 512) {
            umma_bf16_ts_if(leader, d, a, db, idesc_s, c ? 1u : 0u);
            umma_bf16_ts_if(leader, d, a + 8, db + 2, idesc_s, 1u);
            umma_bf16_ts_if(leader, d, a + 16, db + 4, idesc_s, 1u);
            umma_bf16_ts_if(leader, d, a + 24, db + 6, idesc_s, 1u);
          }
          umma_commit_if(leader, &s_full[sb_]);
          if (t == n - 1) umma_commit_if(leader, q_empty);
          ++s_tile;
          if (++s_stage == stages) {
            s_stage = 0;
            s_phase ^= 1;
          }
        }
        if (t > 0) {
          const uint32_t pb = o_tile & 1;
          if (!mbar_wait(&p_full[pb], (o_tile >> 1) & 1, p.status, kStatusTimeoutMma) ||
              (t == 1 && !mbar_wait(o_empty, (piece_no & 1) ^ 1, p.status, kStatusTimeoutMma))) {
            ok = false;
            break;
          }
          tc_fence_after();
          const uint64_t db = dp + pb * p_buf;
          uint64_t da = dt + (uint32_t)o_stage * stage_step;
          uint32_t d = tmem_o;
          const uint32_t more = t > 1 ? 1u : 0u;
#pragma unroll 1
          for (int mc = 0; mc < L.mchunks; ++mc, da += 1024, d += L.hg) {
            umma_bf16_ss_if(leader, d, da, db, idesc_o, more);
            umma_bf16_ss_if(leader, d, da + 128, db + 2, idesc_o, 1u);
            umma_bf16_ss_if(leader, d, da + 256, db + 4, idesc_o, 1u);
            umma_bf16_ss_if(leader, d, da + 384, db + 6, idesc_o, 1u);
          }
          umma_commit_if(leader, &c_empty[o_stage]);
          umma_commit_if(leader, &p_empty[pb]);
          if (t == n) umma_commit_if(leader, o_full);
          ++o_tile;
          if (++o_stage == stages) o_stage = 0;
        }
      }
      cur += n;
    }
  } else if (warp == 0) {
    // ------------------------------ soft-max (thread = head of the group) ------------------------------
    const float scale_log2 = p.scale_log2 * (p.gain ? __bfloat162float(*p.gain) : 1.f);
    uint32_t tn = 0, calls = 0;
    auto waits = [&](uint64_t* bar, uint32_t parity) {
      return __all_sync(0xffffffffu, mbar_wait(bar, parity, p.status, kStatusTimeoutEpilogue)) != 0;
    };
    bool ok = true;
    for (int cur = begin; cur < end && ok;) {
      const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
      const int ctx = p.positions[q.row] + 1;
      const int nh = min(heads_per_group, p.H - q.group * heads_per_group);
      float m_ref = 0.f, l_run = 0.f;
      for (int t = 0; t < q.n; ++t, ++tn) {
        const uint32_t sb_ = tn & 1;
        if (!waits(&s_full[sb_], (tn >> 1) & 1)) {
          ok = false;
          break;
        }
        tc_fence_after();
        float sv[kLBlk];
        {
          uint32_t r0[32], r1[32];
          tmem_ld_32x32(tmem_s + sb_ * 64, r0);
          tmem_ld_32x32(tmem_s + sb_ * 64 + 32, r1);
          tmem_ld_wait();
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&s_empty[sb_]);
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            sv[i] = __uint_as_float(r0[i]) * scale_log2;
            sv[32 + i] = __uint_as_float(r1[i]) * scale_log2;
          }
        }
        const int kv0 = (q.t0 + t) * kLBlk;
        if (kv0 + kLBlk > ctx) {
#pragma unroll
          for (int i = 0; i < kLBlk; ++i)
            if (kv0 + i >= ctx) sv[i] = -INFINITY;
        }
        float m4[4] = {sv[0], sv[1], sv[2], sv[3]};
#pragma unroll
        for (int i = 4; i < kLBlk; ++i) m4[i & 3] = fmaxf(m4[i & 3], sv[i]);
        const float m_tile = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
        if (t == 0) {
          m_ref = m_tile;             // a tile of a row holds at least one visible key
        } else if (__any_sync(0xffffffffu, lane < nh && m_tile > m_ref + 8.f)) {
          // raise the reference maximum: O^T column h times alpha[h], once PV(t - 1) has completed
          const float m_new = fmaxf(m_ref, m_tile);
          const float alpha = fast_exp2(m_ref - m_new);
          m_ref = m_new;
          l_run *= alpha;
          const uint32_t tp = tn - 1;
          if (!waits(&p_empty[tp & 1], (tp >> 1) & 1) || (calls > 0 && !waits(answer, (calls - 1) & 1))) {
            ok = false;
            break;
          }
          s_alpha[lane] = alpha;
          if (lane == 0) *s_call = 0;
          __syncwarp();
          if (lane == 0) mbar_arrive(call);
          if (!waits(answer, calls & 1)) {
            ok = false;
            break;
          }
          ++calls;
        }
        uint32_t pk[kLBlk / 2];
        float rs[2] = {0.f, 0.f};
#pragma unroll
        for (int i = 0; i < kLBlk; i += 2) {
          const float p0 = fast_exp2(sv[i] - m_ref), p1 = fast_exp2(sv[i + 1] - m_ref);
          rs[0] += p0;
          rs[1] += p1;
          pk[i / 2] = pack_bf16x2(p0, p1);
        }
        l_run += rs[0] + rs[1];
        if (!waits(&p_empty[sb_], ((tn >> 1) & 1) ^ 1)) {      // PV(t - 2) has read this buffer
          ok = false;
          break;
        }
        if (lane < L.hg) {
          uint8_t* prow = sP + sb_ * L.hg * 128 + lane * 128;
#pragma unroll
          for (int piece = 0; piece < 8; ++piece) {
            uint4 v = make_uint4(pk[piece * 4], pk[piece * 4 + 1], pk[piece * 4 + 2], pk[piece * 4 + 3]);
            if (lane >= nh) v = make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint4*>(prow + ((piece ^ (lane & 7)) << 4)) = v;
          }
        }
        fence_proxy_async_smem();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[sb_]);
      }
      if (!ok) break;
      // hand the statistics over and go on: the result is written while the next piece's first tiles are under way
      if (calls > 0 && !waits(answer, (calls - 1) & 1)) break;
      s_l[lane] = 1.f / l_run;      // l_run is at least one: a row's maximum has weight one
      s_m[lane] = m_ref + log2f(l_run);
      if (lane == 0) *s_call = 1;
      __syncwarp();
      if (lane == 0) mbar_arrive(call);
      ++calls;
      cur += q.n;
    }
  } else if (warp <= 4) {
    // ------------------------------ O^T: rescaling and output (warp 4: rows 0..31, warps 1..3: the others) ----------------
    const int quarter = warp & 3;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    const int col0 = quarter * 32 + lane;
    uint32_t calls = 0, piece_no = 0;
    for (int cur = begin; cur < end;) {
      if (!__all_sync(0xffffffffu, mbar_wait(call, calls & 1, p.status, kStatusTimeoutEpilogue))) break;
      ++calls;
      if (*s_call == 0) {
        tc_fence_after();
#pragma unroll 1
        for (int mc = 0; mc < L.mchunks; ++mc)
#pragma unroll 1
          for (int c = 0; c < L.hg; c += 16) {
            uint32_t r[16];
            tmem_ld_32x16(tmem_o + lane_off + mc * L.hg + c, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * s_alpha[c + i]);
            tmem_st_32x16(tmem_o + lane_off + mc * L.hg + c, r);
          }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(answer);
        continue;
      }
      const LdPiece q = ld_piece(s_pre, p.T, L.groups, cur, end);
      const int head0 = q.group * heads_per_group;
      const int nh = min(heads_per_group, p.H - head0);
      if (!__all_sync(0xffffffffu, mbar_wait(o_full, piece_no & 1, p.status, kStatusTimeoutEpilogue))) break;
      tc_fence_after();
      const int slot = 2 * blockIdx.x + (cur == begin ? 0 : 1);
      __nv_bfloat16* orow = p.out + ((size_t)q.row * p.H + head0) * p.R + col0;
      float* wrow = p.ws_o + (size_t)slot * L.hg * p.R + col0;
#pragma unroll 1
      for (int mc = 0; mc < L.mchunks; ++mc) {
        const bool in = mc * 128 + col0 < p.R;
#pragma unroll 1
        for (int c = 0; c < nh; c += 16) {
          uint32_t r[16];
          tmem_ld_32x16(tmem_o + lane_off + mc * L.hg + c, r);
          tmem_ld_wait();
          const size_t at = (size_t)c * p.R + mc * 128;
          float v[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]) * s_l[c + i];
          if (q.whole) {
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (in && c + i < nh) orow[at + (size_t)i * p.R] = __float2bfloat16(v[i]);
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (in && c + i < nh) wrow[at + (size_t)i * p.R] = v[i];
          }
        }
      }
      if (!q.whole && warp == 4 && lane < nh) p.ws_lse[(size_t)slot * L.hg + lane] = s_m[lane];
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(o_empty);
        mbar_arrive(answer);
      }
      ++piece_no;
      cur += q.n;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 6) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

// rows whose tiles are spread over several CTAs: weighted mean of the partial results; zero rows for idle slots
constexpr int kLMaxGrid = 256;
__global__ void __launch_bounds__(128) latent_merge_kernel(LdParams p, int hg, int groups, int grid) {
  __shared__ float s_w[kLMaxGrid];
  __shared__ int s_at[kLMaxGrid];
  __shared__ float s_red[8];
  const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int per_group = (p.H + groups - 1) / groups, group = h / per_group;
  const int before = p.ws_pre[row], tiles = p.ws_pre[row + 1] - before;
  __nv_bfloat16* orow = p.out + ((size_t)row * p.H + h) * p.R;
  if (tiles == 0) {
    for (int d = tid; d < p.R; d += 128) orow[d] = __float2bfloat16(0.f);
    return;
  }
  const long long total = (long long)p.ws_pre[p.T] * groups;
  const long long s0 = (long long)before * groups + (long long)group * tiles, s1 = s0 + tiles - 1;
  const int c0 = (int)(((s0 + 1) * grid - 1) / total), c1 = (int)(((s1 + 1) * grid - 1) / total);
  if (c0 == c1) return;
  const int n = c1 - c0 + 1;
  // piece j lies in CTA c0 + j: its place in the workspace and its weight (a CTA without tiles has none)
  float m = -INFINITY;
  for (int j = tid; j < n; j += 128) {
    const int c = c0 + j, b = ld_range(total, c, grid);
    const bool none = b == ld_range(total, c + 1, grid);
    const int at = (2 * c + (j == 0 && b != s0 ? 1 : 0)) * hg + h - group * per_group;
    s_at[j] = at;
    s_w[j] = none ? -INFINITY : p.ws_lse[at];
    m = fmaxf(m, s_w[j]);
  }
  m = warp_max(m);
  if ((tid & 31) == 0) s_red[tid >> 5] = m;
  __syncthreads();
  m = fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3]));
  float sum = 0.f;
  for (int j = tid; j < n; j += 128) {
    s_w[j] = fast_exp2(s_w[j] - m);
    sum += s_w[j];
  }
  sum = warp_sum(sum);
  if ((tid & 31) == 0) s_red[4 + (tid >> 5)] = sum;
  __syncthreads();
  const float inv = 1.f / (s_red[4] + s_red[5] + s_red[6] + s_red[7]);
  for (int d = tid * 4; d < p.R; d += 512) {      // R is a multiple of eight
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int j = 0; j < n; ++j) {
      const float w = s_w[j];
      if (w == 0.f) continue;
      const float4 v = *reinterpret_cast<const float4*>(p.ws_o + (size_t)s_at[j] * p.R + d);
      acc.x = fmaf(w, v.x, acc.x);
      acc.y = fmaf(w, v.y, acc.y);
      acc.z = fmaf(w, v.z, acc.z);
      acc.w = fmaf(w, v.w, acc.w);
    }
    *reinterpret_cast<uint2*>(orow + d) = make_uint2(pack_bf16x2(acc.x * inv, acc.y * inv), pack_bf16x2(acc.z * inv, acc.w * inv));
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
  return L.stages >= 2 ? L.groups : 0;
}

extern "C" int sb_latent_decode_grid() { return num_sms() < kLMaxGrid ? num_sms() : kLMaxGrid; }

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
  CUtensorMap mc;
  int r = make_tensor_map_bf16_3d(&mc, w.cache, w.R, kLBlk, w.num_blocks, w.R, (long long)kLBlk * w.R, 64, kLBlk, 1);
  if (r) return r;
  const int grid = sb_latent_decode_grid();
  LdParams p;
  p.seq_ids = w.seq_ids; p.positions = w.positions; p.block_table = w.block_table; p.num_blocks = w.num_blocks;
  p.max_blocks = w.max_blocks; p.T = w.T; p.H = w.H; p.R = w.R;
  p.scale_log2 = w.scale * 1.4426950408889634f;
  p.gain = reinterpret_cast<const __nv_bfloat16*>(w.gain);
  p.qa = reinterpret_cast<const __nv_bfloat16*>(w.qa);
  p.out = reinterpret_cast<__nv_bfloat16*>(w.out);
  p.ws_o = ws_o; p.ws_lse = ws_stat; p.ws_pre = reinterpret_cast<int*>(ws_stat + (size_t)2 * grid * L.hg);
  p.status = status;
  static int configured = 0;
  if (configured < L.total) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total);
    if (e != cudaSuccess) return (int)e;
    configured = L.total;
  }
  latent_decode_kernel<<<grid, 288, L.total, stream>>>(mc, p);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  latent_merge_kernel<<<dim3(w.T, w.H), 128, 0, stream>>>(p, L.hg, L.groups, grid);
  return (int)cudaGetLastError();
}
