// Shared by the kernels of the matrix-state recurrences (linear_scan.cu, linear_chunk.cu).
#pragma once

#include "fr_common.cuh"

namespace fr {
namespace scan {

// Layout of one head's state: [rows][cols] fp32, both padded with zeros.
__host__ __device__ __forceinline__ int state_rows(int dim) { return (dim + 7) / 8 * 8; }
__host__ __device__ __forceinline__ int state_cols(int vdim) { return (vdim + 15) / 16 * 16; }

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void from_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// two fp32 operations per instruction
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ uint64_t dup2(float v) { return pack2(v, v); }
__device__ __forceinline__ void unpack2(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// FR_DECAY_CHANNEL: log sigmoid(bias + up . low) / tau of channel `ch` (head * dim + dimension)
__device__ __forceinline__ float channel_log_decay(const fr_linear_scan& a, int64_t t, int ch) {
  float z = a.step_bias[ch];
  const float* low = a.step + t * a.ldstep;
  const float* up = a.up + static_cast<int64_t>(ch) * a.rank;
  for (int i = 0; i < a.rank; ++i) z = fmaf(up[i], low[i], z);
  return -softplus(-z) * a.inv_tau;
}
// FR_DECAY_HEAD: step size of a head, softplus(step + bias)
__device__ __forceinline__ float head_step(const fr_linear_scan& a, int64_t t, int h) {
  return softplus(a.step[t * a.ldstep + h] + a.step_bias[h]);
}

// linear_scan.cu: the heads [request, head] with a flag, of requests of at least min_tokens tokens (bf16, decay per channel)
int rows_flagged(const fr_linear_scan& a, int n_req, int min_tokens, const int32_t* flags, cudaStream_t stream);

static inline int check_args(const fr_linear_scan* a) {
  FR_CHECK_ARG(a && (a->dtype == 0 || a->dtype == 1) && (a->decay == FR_DECAY_CHANNEL || a->decay == FR_DECAY_HEAD));
  FR_CHECK_ARG(a->heads > 0 && a->heads <= 65535 && a->key_heads > 0 && a->heads % a->key_heads == 0 && a->dim > 0 && a->vdim > 0);
  FR_CHECK_ARG(a->q && a->k && a->v && a->out && a->step && a->step_bias && a->state && a->state_slots && a->qo_indptr && a->pos);
  FR_CHECK_ARG(a->decay == FR_DECAY_HEAD ? a->rate != nullptr : (a->up != nullptr && a->rank > 0 && a->key_heads == a->heads));
  FR_CHECK_ARG((reinterpret_cast<uintptr_t>(a->state) & 15u) == 0);
  return FR_OK;
}

}  // namespace scan
}  // namespace fr
