// Every head's rows times the head's own matrix (latent_params.h): the key and value expansions of latent attention folded
// into the query and the output of a decoding step.
//
//   head_product_kernel   bf16 on tcgen05: one CTA per (128 columns, head, 128 rows).  A rows, one head's columns, come by
//                         TMA through a three-dimensional map (columns past the head's width are zeros); B_h is read as it
//                         is stored, K-major or through an MN-major descriptor, so both expansions use the checkpoint's
//                         layout.  The output gate is applied in the epilogue.
//   head_product_simt     fp32, and bf16 of any size
#include "common.cuh"
#include "launchers.h"
#include "latent_params.h"
#include "typed.cuh"

namespace sb {

constexpr int kHpBytes = 128 * 64 * 2;     // one operand tile of a stage: 128 rows or columns x 64 of the contraction

// few wide tiles with a short contraction (queries) keep two CTAs on an SM; a long contraction gets a deep ring
template <bool B_MN>
struct HpSmem {
  static constexpr int kStages = B_MN ? 3 : 6;
  static constexpr int kBarOff = kStages * 2 * kHpBytes;
  static constexpr int kTotal = kBarOff + (2 * kStages + 1) * 8 + 16 + 1024;
};

template <bool B_MN>
__global__ void __launch_bounds__(192)
head_product_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b, HeadProduct p,
                    int* status) {
  constexpr int kHpStages = HpSmem<B_MN>::kStages;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + HpSmem<B_MN>::kBarOff);
  uint64_t* empty = full + kHpStages;
  uint64_t* done = empty + kHpStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * 128, h = blockIdx.y, m0 = blockIdx.z * 128;
  const int N = B_MN ? p.b_cols : p.b_rows, K = B_MN ? p.b_rows : p.b_cols;
  const int nk = (K + 63) / 64;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&map_a);
    tma_prefetch_desc(&map_b);
    for (int s = 0; s < 2 * kHpStages + 1; ++s) mbar_init(&full[s], 1);
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 128);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      int k = 0;
      for (; k < nk; ++k) {
        const int s = k % kHpStages;
        if (!mbar_wait(&empty[s], ((k / kHpStages) & 1) ^ 1, status, kStatusTimeoutProducer)) {
          ok = false;
          break;
        }
        uint8_t* sa = smem + s * 2 * kHpBytes;
        uint8_t* sb_ = sa + kHpBytes;
        mbar_arrive_expect_tx(&full[s], 2 * kHpBytes);
        tma_load_3d(sa, &map_a, &full[s], k * 64, h, m0);
        if constexpr (B_MN) {
          tma_load_3d(sb_, &map_b, &full[s], n0, k * 64, h);
          tma_load_3d(sb_ + 8192, &map_b, &full[s], n0 + 64, k * 64, h);
        } else {
          tma_load_3d(sb_, &map_b, &full[s], k * 64, n0, h);
        }
      }
      if (!ok)      // no copy may be in flight when shared memory is given back
        for (int j = (k > kHpStages ? k - kHpStages : 0); j < k; ++j)
          mbar_wait(&full[j % kHpStages], (j / kHpStages) & 1, nullptr, 0);
    }
  } else if (warp == 1) {
    constexpr uint32_t idesc = umma_idesc_bf16(128, 128, 0, B_MN ? 1 : 0);
    bool ok = true;
    for (int k = 0; k < nk && ok; ++k) {
      const int s = k % kHpStages;
      ok = mbar_wait(&full[s], (k / kHpStages) & 1, status, kStatusTimeoutMma);
      if (!ok) break;
      tc_fence_after();
      if (lane == 0) {
        const uint32_t sa = smem_u32(smem + s * 2 * kHpBytes), sb_ = sa + kHpBytes;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          const uint64_t da = umma_smem_desc(sa + kk * 32, 16, 1024);
          const uint64_t db = B_MN ? umma_smem_desc(sb_ + kk * 2048, 8192, 1024) : umma_smem_desc(sb_ + kk * 32, 16, 1024);
          umma_bf16_ss(tmem, da, db, idesc, (k | kk) ? 1u : 0u);
        }
        umma_commit(&empty[s]);
      }
      __syncwarp();
    }
    if (ok && lane == 0) umma_commit(done);
    __syncwarp();
  } else {
    const int quarter = warp & 3, row = m0 + quarter * 32 + lane;
    const bool valid = row < p.T;
    const long long col0 = (long long)h * N + n0;
    const float gain = p.gain ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(p.gain)) : 1.f;
    // the gate's row is fetched while the product runs
    uint4 g[16];
    const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(p.gate) + (long long)(valid ? row : 0) * p.gate_row + col0;
#pragma unroll
    for (int v = 0; v < 16; ++v)
      if (p.gate && valid && n0 + v * 8 < N) g[v] = *reinterpret_cast<const uint4*>(gate + v * 8);
    if (__all_sync(0xffffffffu, mbar_wait(done, 0, status, kStatusTimeoutEpilogue))) {
      tc_fence_after();
      __nv_bfloat16* c = reinterpret_cast<__nv_bfloat16*>(p.c) + (long long)(valid ? row : 0) * p.c_row + col0;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (n0 + q * 32 >= N) break;
        uint32_t r[32];
        tmem_ld_32x32(tmem + ((uint32_t)(quarter * 32) << 16) + q * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int v = 0; v < 4; ++v) {
          if (!valid || n0 + q * 32 + v * 8 >= N) break;
          float o[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) o[i] = __uint_as_float(r[v * 8 + i]);
          if (p.gate) {
            const __nv_bfloat162* z2 = reinterpret_cast<const __nv_bfloat162*>(&g[q * 4 + v]);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const float2 z = __bfloat1622float2(z2[i]);
              o[2 * i] = __fdividef(o[2 * i], 1.f + __expf(-gain * z.x));
              o[2 * i + 1] = __fdividef(o[2 * i + 1], 1.f + __expf(-gain * z.y));
            }
          }
          store_vec<__nv_bfloat16, 8>(c + q * 32 + v * 8, o);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 128);
  }
}

// 64 x 64 output tile of one head per 256 threads, 4 x 4 values each
template <typename T>
__global__ void __launch_bounds__(256) head_product_simt(HeadProduct p) {
  __shared__ float sa[16][68], sb_[16][68];
  const int n0 = blockIdx.x * 64, h = blockIdx.y, m0 = blockIdx.z * 64;
  const int N = p.b_mn ? p.b_cols : p.b_rows, K = p.b_mn ? p.b_rows : p.b_cols;
  const long long bn = p.b_mn ? 1 : p.b_cols, bk = p.b_mn ? p.b_cols : 1;
  const T* A = reinterpret_cast<const T*>(p.a) + h * p.a_head;
  const T* B = reinterpret_cast<const T*>(p.b) + (long long)h * p.b_rows * p.b_cols;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i >> 4, k = i & 15;
      sa[k][r] = (m0 + r < p.T && k0 + k < K) ? to_float(A[(m0 + r) * p.a_row + k0 + k]) : 0.f;
      // consecutive threads walk the contiguous direction of B
      const int rn = p.b_mn ? i & 63 : r, kn = p.b_mn ? i >> 6 : k;
      sb_[kn][rn] = (n0 + rn < N && k0 + kn < K) ? to_float(B[(n0 + rn) * bn + (k0 + kn) * bk]) : 0.f;
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
  const float gain = p.gain ? to_float(*reinterpret_cast<const T*>(p.gain)) : 1.f;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= p.T || n >= N) continue;
      float v = acc[i][j];
      if (p.gate)
        v /= 1.f + expf(-gain * to_float(reinterpret_cast<const T*>(p.gate)[m * p.gate_row + (long long)h * N + n]));
      reinterpret_cast<T*>(p.c)[m * p.c_row + (long long)h * N + n] = from_float<T>(v);
    }
}

}  // namespace sb

using namespace sb;

extern "C" int sb_head_product_simt(const void* params, int f32, cudaStream_t stream) {
  HeadProduct p = *reinterpret_cast<const HeadProduct*>(params);
  if (p.T <= 0) return 0;
  if (p.H > 65535) return -3;
  const int N = p.b_mn ? p.b_cols : p.b_rows;
  const int esize = f32 ? 4 : 2;
  auto shift = [&](const void* q, long long n) { return reinterpret_cast<const char*>(q) + n * esize; };
  const int all = p.T, most = 64 * 65535;
  for (int s = 0; s < all; s += most) {
    HeadProduct q = p;
    q.T = all - s < most ? all - s : most;
    q.a = shift(p.a, s * p.a_row);
    q.c = const_cast<char*>(shift(p.c, s * p.c_row));
    if (p.gate) q.gate = shift(p.gate, s * p.gate_row);
    const dim3 grid((N + 63) / 64, p.H, (q.T + 63) / 64);
    if (f32) head_product_simt<float><<<grid, 256, 0, stream>>>(q);
    else head_product_simt<__nv_bfloat16><<<grid, 256, 0, stream>>>(q);
  }
  return (int)cudaGetLastError();
}

extern "C" int sb_head_product(const void* params, int* status, cudaStream_t stream) {
  const HeadProduct& p = *reinterpret_cast<const HeadProduct*>(params);
  if (p.T <= 0) return 0;
  const int N = p.b_mn ? p.b_cols : p.b_rows, K = p.b_mn ? p.b_rows : p.b_cols;
  if (p.H > 65535 || p.T > 128 * 65535 || N % 8 || p.b_cols % 8 || p.a_head % 8 || p.a_row % 8 || p.c_row % 8 ||
      p.gate_row % 8 || ((uintptr_t)p.a & 15) || ((uintptr_t)p.b & 15) || ((uintptr_t)p.c & 15) || ((uintptr_t)p.gate & 15))
    return -3;
  static thread_local bool tl_context_bound = false;
  if (!tl_context_bound) {
    cudaFree(0);
    tl_context_bound = true;
  }
  CUtensorMap ma, mb;
  int r = make_tensor_map_bf16_3d(&ma, p.a, K, p.H, p.T, p.a_head, p.a_row, 64, 1, 128);
  if (r) return r;
  r = make_tensor_map_bf16_3d(&mb, p.b, p.b_cols, p.b_rows, p.H, p.b_cols, (long long)p.b_rows * p.b_cols, 64,
                              p.b_mn ? 64 : 128, 1);
  if (r) return r;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(head_product_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         HpSmem<true>::kTotal);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(head_product_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                               HpSmem<false>::kTotal);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((N + 127) / 128, p.H, (p.T + 127) / 128);
  if (p.b_mn) head_product_kernel<true><<<grid, 192, HpSmem<true>::kTotal, stream>>>(ma, mb, p, status);
  else head_product_kernel<false><<<grid, 192, HpSmem<false>::kTotal, stream>>>(ma, mb, p, status);
  return (int)cudaGetLastError();
}
