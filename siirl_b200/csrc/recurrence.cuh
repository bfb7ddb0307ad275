// What the kernels of the matrix-state recurrences share (recurrence.cu, delta_rule.cu): arguments, gates, fragments of the
// tensor cores' warp-level products, asynchronous copies.
#pragma once
#include "common.cuh"
#include "launchers.h"
#include "typed.cuh"

namespace sb {

enum { kGateChannel = 0, kGateHead = 1, kGateDelta = 2 };
constexpr int kChunk = 16;
constexpr float kLog2e = 1.4426950408889634f;

struct RecParams {
  const void* x;               // projected rows [T, row_stride]
  long long row_stride;
  int q_off, k_off, v_off, g_off;
  int e_off, f_off;            // kGateChannel: low-rank row at e_off; kGateHead: i_pre at e_off, f_pre at f_off (per head);
                               // kGateDelta: low-rank row at e_off, pre-activations of the removal rates at f_off
  int kind, rank, norm_per_head, gate_act;   // gate_act: 0 SiLU, 1 sigmoid
  const void* w2;              // [H * dk, rank]
  const void* b_e;             // kGateChannel, kGateDelta: [H * dk]; kGateHead: input-gate bias [H]
  const void* b_f;             // kGateHead: forget-gate bias [H]; kGateDelta: bias of the removal rates [H * dk]
  const void* norm_w;
  float inv_tau, cap, q_scale, eps, out_scale;
  float* S;
  float* m;
  void* out;                   // [T, out_stride], this branch at column out_off
  long long out_stride;
  int out_off, H, dk, dv;
};

static_assert(sizeof(RecParams) == 160, "RecParams is mirrored by a ctypes structure in ops/recurrence.py");

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gate_value(float g, int act) {
  const float s = 1.f / (1.f + expf(-g));
  return act == 0 ? g * s : s;
}
__device__ __forceinline__ float fast_gate(float g, int act) {
  const float s = __fdividef(1.f, 1.f + __expf(-g));
  return act == 0 ? g * s : s;
}
constexpr int kStepThreads = 256;
// key channels padded to a width the scan is compiled for: 16, 32, 48, 64, 96 or 128
__host__ __device__ inline int pad_dk(int dk) { return dk <= 64 ? (dk + 15) / 16 * 16 : (dk + 31) / 32 * 32; }
__host__ __device__ inline int tile_row(int dkp) { return dkp + 8; }        // bf16 elements per row of a q / k tile
constexpr int kARow = 24;                                                    // and of the score matrix

// runs of consecutive chunks of one sequence
struct Segments {
  const int* seq;       // [n] sequence of the segment
  const int* chunk0;    // [n] its first chunk
  const int* row;       // [n] its first row
  const int* tokens;    // [n] its tokens
  const int* flags;     // [n] bit 0: first of its sequence, bit 1: last
  const int* seq_seg0;  // [n_seq + 1]
  float* S;             // [n, H, rows, dk] local states, then start states
  float* decay;         // [n, H, dkp] (kGateDelta: [n, H, dk, dk], what a start state is multiplied by)
};

// x and y as two bf16 terms each: x = hi + lo to 16 mantissa bits
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16x2(x - f.x, y - f.y);
}

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace sb
