// Row kernels of the 16/32-bit decoder layers: embedding lookup into the fp32 residual stream (with the slot
// table entry of every new token), RMS norm of the fp32 stream, updates of the stream by normalised vectors fused with
// the norm that follows, gated norms over groups of columns, norm and rotation of queries and keys, and the short
// causal convolution with its state.
#include "fr_common.cuh"
#include "sm100_ptx.cuh"

namespace fr {
namespace lm {

template <typename T>
__device__ __forceinline__ float ld_f(const T* p) { return static_cast<float>(*p); }
template <>
__device__ __forceinline__ float ld_f<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T>
__device__ __forceinline__ void st_f(T* p, float v) { *p = v; }
template <>
__device__ __forceinline__ void st_f<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

template <typename T>
__global__ void __launch_bounds__(256)
embed_kernel(const T* __restrict__ table, int64_t ldt, const int64_t* __restrict__ ids, float* __restrict__ x, int64_t ldx, int W,
             int vocab, float scale, int32_t* __restrict__ req_to_token, int64_t table_stride,
             const int64_t* __restrict__ rows, const int64_t* __restrict__ pos, const int64_t* __restrict__ loc) {
  const int64_t t = blockIdx.x;
  int64_t id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + id * ldt;
  for (int c = threadIdx.x; c < W; c += blockDim.x) x[t * ldx + c] = ld_f(src + c) * scale;
  if (req_to_token != nullptr && threadIdx.x == 0)
    req_to_token[rows[t] * table_stride + pos[t]] = static_cast<int32_t>(loc[t]);
}

// One CTA per row; a row is read once into registers (up to 8 float4 per thread) or, when wider, re-read.
constexpr int kNormThreads = 256;
constexpr int kNormVec = 8;

template <typename T, bool VEC>
__global__ void __launch_bounds__(kNormThreads)
norm_kernel(float* __restrict__ x, int64_t ldx, const float* __restrict__ weight, float offset, float eps,
            const float* __restrict__ partials, int n_partials, int64_t partial_stride,
            const int64_t* __restrict__ row_idx, T* __restrict__ out, int64_t ldo, int W) {
  __shared__ float warp_sums[kNormThreads / 32];
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t t = blockIdx.x;
  const int64_t src = row_idx != nullptr ? row_idx[t] : t;
  float* xr = x + src * ldx;
  T* o = out + t * ldo;
  const float* pr = partials != nullptr ? partials + src * W : nullptr;
  // one element with its partials, in order (scalar path)
  auto value = [&](int c) {
    float f = xr[c];
    if (pr != nullptr)
      for (int s = 0; s < n_partials; ++s) f += pr[s * partial_stride + c];
    return f;
  };
  float ss = 0.f;
  float4 v[kNormVec];
  if constexpr (VEC) {
#pragma unroll
    for (int i = 0; i < kNormVec; ++i) {
      const int c = (i * kNormThreads + threadIdx.x) * 4;
      v[i] = make_float4(0, 0, 0, 0);
      if (c < W) {
        v[i] = *reinterpret_cast<const float4*>(xr + c);
        if (pr != nullptr) {
          for (int s = 0; s < n_partials; ++s) {
            const float4 p = *reinterpret_cast<const float4*>(pr + s * partial_stride + c);
            v[i].x += p.x; v[i].y += p.y; v[i].z += p.z; v[i].w += p.w;
          }
          if (row_idx == nullptr) *reinterpret_cast<float4*>(xr + c) = v[i];
        }
        ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
      }
    }
  } else {
    for (int c = threadIdx.x; c < W; c += kNormThreads) {
      const float f = value(c);
      ss += f * f;
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) warp_sums[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < kNormThreads / 32; ++i) tot += warp_sums[i];
  const float r = 1.0f / sqrtf(tot / static_cast<float>(W) + eps);
  if constexpr (VEC) {
#pragma unroll
    for (int i = 0; i < kNormVec; ++i) {
      const int c = (i * kNormThreads + threadIdx.x) * 4;
      if (c < W) {
        const float4 w = *reinterpret_cast<const float4*>(weight + c);
        const float a = v[i].x * r * (offset + w.x), b = v[i].y * r * (offset + w.y);
        const float d = v[i].z * r * (offset + w.z), e = v[i].w * r * (offset + w.w);
        if constexpr (sizeof(T) == 2) {
          *reinterpret_cast<uint2*>(o + c) = make_uint2(pack_bf16(a, b), pack_bf16(d, e));
        } else {
          *reinterpret_cast<float4*>(o + c) = make_float4(a, b, d, e);
        }
      }
    }
  } else {
    for (int c = threadIdx.x; c < W; c += kNormThreads) {
      const float f = value(c);
      st_f(o + c, f * r * (offset + weight[c]));
      if (pr != nullptr && row_idx == nullptr) xr[c] = f;
    }
  }
  const int wpad = (W + 7) / 8 * 8;
  for (int c = W + threadIdx.x; c < wpad && c < ldo; c += kNormThreads) st_f(o + c, 0.f);
}

struct ConvOuts {
  fr_conv_out o[4];
  int n;
  const float* bias;
  int act;  // fr_conv_act
};

// silu; the 16-bit results leave through a fast exponential
template <typename T>
__device__ __forceinline__ float silu_t(float z) {
  return sizeof(T) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));
}

// Value of channel c at `back` tokens before token t of the batch (e = index of t within its request).
template <typename T>
__device__ __forceinline__ float conv_tap(const T* __restrict__ u, int64_t ldu, const T* __restrict__ st, int C, int taps, int64_t t,
                                          int e, int64_t pos, int c, int back) {
  if (pos < back) return 0.f;
  if (e >= back) return ld_f(u + (t - back) * ldu + c);
  return ld_f(st + static_cast<int64_t>(taps - 1 + e - back) * C + c);
}

// Eight channels per thread, 16-byte accesses. ONE: one token per request (and per blockIdx.x). Otherwise a thread
// walks up to kConvRun consecutive tokens with the window of past values in registers; it reloads the window where
// another request begins.
constexpr int kConvRun = 16;

// eight consecutive values as they lie in memory
template <typename T>
struct Raw8 {
  uint4 q[sizeof(T) / 2];
};
template <typename T>
__device__ __forceinline__ Raw8<T> raw_load(const T* p) {
  Raw8<T> r;
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T)) / 2; ++i) r.q[i] = reinterpret_cast<const uint4*>(p)[i];
  return r;
}
template <typename T>
__device__ __forceinline__ void raw_store(T* p, const Raw8<T>& r) {
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T)) / 2; ++i) reinterpret_cast<uint4*>(p)[i] = r.q[i];
}
template <typename T>
__device__ __forceinline__ Raw8<T> raw_zero() {
  Raw8<T> r;
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T)) / 2; ++i) r.q[i] = make_uint4(0, 0, 0, 0);
  return r;
}
__device__ __forceinline__ void raw_unpack(const Raw8<float>& r, float (&v)[8]) {
  const uint32_t w[8] = {r.q[0].x, r.q[0].y, r.q[0].z, r.q[0].w, r.q[1].x, r.q[1].y, r.q[1].z, r.q[1].w};
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(w[i]);
}
__device__ __forceinline__ void raw_unpack(const Raw8<__nv_bfloat16>& r, float (&v)[8]) {
  const uint32_t w[4] = {r.q[0].x, r.q[0].y, r.q[0].z, r.q[0].w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
template <typename T>
__device__ __forceinline__ void conv_store8(T* p, const float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) =
        make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
}

template <typename T, int TAPS, bool ONE>
__global__ void __launch_bounds__(128)
conv_vec_kernel(const T* __restrict__ u, int64_t ldu, const float* __restrict__ w, int C, const __grid_constant__ ConvOuts outs,
                T* __restrict__ state, const int64_t* __restrict__ state_slots, const int32_t* __restrict__ tok_req,
                const int32_t* __restrict__ qo_indptr, const int64_t* __restrict__ pos, int n_tok) {
  constexpr int P = TAPS - 1;
  const int c = (blockIdx.y * 128 + threadIdx.x) * 8;
  float wr[TAPS][8];
  if (c < C) {
    float flat[8 * TAPS];  // TAPS * 8 consecutive values
#pragma unroll
    for (int i = 0; i < 2 * TAPS; ++i) {
      const float4 q = __ldg(reinterpret_cast<const float4*>(w + static_cast<int64_t>(c) * TAPS) + i);
      flat[4 * i] = q.x; flat[4 * i + 1] = q.y; flat[4 * i + 2] = q.z; flat[4 * i + 3] = q.w;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int k = 0; k < TAPS; ++k) wr[k][i] = flat[i * TAPS + k];
  }
  float b0[8] = {};
  if (c < C && outs.bias != nullptr)
#pragma unroll
    for (int i = 0; i < 8; ++i) b0[i] = outs.bias[c + i];
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  if (c >= C) return;
  int oi = 0;
  while (oi + 1 < outs.n && !(c >= outs.o[oi].c0 && c < outs.o[oi].c0 + outs.o[oi].c)) ++oi;
  const fr_conv_out& o = outs.o[oi];
  const bool keep = c >= o.c0 && c < o.c0 + o.c;
  T* out = static_cast<T*>(o.out) + (c - o.c0);
  Raw8<T> win[P];
  const int t0 = ONE ? blockIdx.x : blockIdx.x * kConvRun;
  const int t1 = ONE ? t0 + 1 : min(t0 + kConvRun, n_tok);
  constexpr int B = ONE ? 1 : 4;  // tokens loaded together, the next ones while these are worked on
  Raw8<T> v[B], nv[B];
  int req[B], nreq[B];
  int64_t dst[B], ndst[B];
  auto fetch = [&](int t) {
#pragma unroll
    for (int i = 0; i < B; ++i)
      if (t + i < t1) {
        nv[i] = raw_load<T>(u + static_cast<int64_t>(t + i) * ldu + c);
        nreq[i] = tok_req[t + i];
        ndst[i] = o.row_map != nullptr ? o.row_map[t + i] : t + i;
      }
  };
  int cur = -1;
  fetch(t0);
#pragma unroll
  for (int k = 0; k < P; ++k) win[k] = raw_zero<T>();
  if (!ONE) {  // the tokens just before the run are the window when they belong to the same request
    bool same = t0 >= P;
    if (same) {
      const int b0 = tok_req[t0];
#pragma unroll
      for (int k = 0; k < P; ++k) {
        win[k] = raw_load<T>(u + static_cast<int64_t>(t0 - (P - k)) * ldu + c);
        same = same && tok_req[t0 - (P - k)] == b0;
      }
      if (same) cur = b0;
    }
  }
  for (int t = t0; t < t1; t += B) {
#pragma unroll
    for (int x = 0; x < B; ++x) {
      v[x] = nv[x];
      req[x] = nreq[x];
      dst[x] = ndst[x];
    }
    if (t + B < t1) fetch(t + B);
#pragma unroll
    for (int x = 0; x < B; ++x) {
      if (t + x >= t1) break;
      const int b = req[x];
      if (b != cur) {  // fill the window: earlier tokens of the batch, then the state, zeros before position 0
        cur = b;
        const int64_t p = pos[t + x];
        const int e = ONE ? 0 : t + x - qo_indptr[b];
        const T* st = state + state_slots[b] * P * C + c;
#pragma unroll
        for (int k = 0; k < P; ++k) {
          const int back = P - k;
          if (p < back) {
            win[k] = raw_zero<T>();
          } else if (e >= back) {
            win[k] = raw_load<T>(u + static_cast<int64_t>(t + x - back) * ldu + c);
          } else {
            win[k] = raw_load<T>(st + static_cast<int64_t>(k + e) * C);
          }
        }
      }
      float y[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = b0[i];
#pragma unroll
      for (int k = 0; k < TAPS; ++k) {
        float f[8];
        raw_unpack(k < P ? win[k < P ? k : 0] : v[x], f);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(wr[k][i], f[i], y[i]);
      }
      if (outs.act == FR_CONV_SILU)
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = silu_t<T>(y[i]);
      if (keep) conv_store8<T>(out + dst[x] * o.ldo, y);
#pragma unroll
      for (int k = 0; k + 1 < P; ++k) win[k] = win[k + 1];
      win[P - 1] = v[x];
      if (ONE) {  // the window is the request's new state
        T* st = state + state_slots[b] * P * C + c;
#pragma unroll
        for (int k = 0; k < P; ++k) raw_store<T>(st + static_cast<int64_t>(k) * C, win[k]);
      }
    }
  }
}

// One token and 256 channels per CTA. ONE: every request has one token, so the thread that has read a channel's
// state also advances it.
template <typename T, bool ONE>
__global__ void __launch_bounds__(256)
short_conv_kernel(const T* __restrict__ u, int64_t ldu, const float* __restrict__ w, int taps, int C,
                  const __grid_constant__ ConvOuts outs, T* __restrict__ state, const int64_t* __restrict__ state_slots,
                  const int32_t* __restrict__ tok_req, const int32_t* __restrict__ qo_indptr,
                  const int64_t* __restrict__ pos) {
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t t = blockIdx.x;
  const int c = blockIdx.y * 256 + threadIdx.x;
  if (c >= C) return;
  const int b = tok_req[t];
  const int e = ONE ? 0 : static_cast<int>(t - qo_indptr[b]);
  const int64_t p = pos[t];
  T* st = state + state_slots[b] * (taps - 1) * C;
  const float* wc = w + static_cast<int64_t>(c) * taps;
  float y = outs.bias != nullptr ? outs.bias[c] : 0.f;
  for (int back = taps - 1; back >= 0; --back)
    y = fmaf(wc[taps - 1 - back], conv_tap(u, ldu, st, C, taps, t, e, p, c, back), y);
  if (outs.act == FR_CONV_SILU) y = silu_t<T>(y);
  for (int i = 0; i < outs.n; ++i) {
    const fr_conv_out& o = outs.o[i];
    if (c >= o.c0 && c < o.c0 + o.c) {
      const int64_t r = o.row_map != nullptr ? o.row_map[t] : t;
      st_f(static_cast<T*>(o.out) + r * o.ldo + (c - o.c0), y);
    }
  }
  if (ONE) {
    for (int i = 0; i + 1 < taps - 1; ++i) st[static_cast<int64_t>(i) * C + c] = st[static_cast<int64_t>(i + 1) * C + c];
    if (taps > 1) st[static_cast<int64_t>(taps - 2) * C + c] = u[t * ldu + c];
  }
}

// The last taps - 1 values of every request after this batch; entry i comes from local index n - (taps - 1) + i,
// negative indices from the old state (always a later entry, so ascending order may overwrite in place).
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const T* __restrict__ u, int64_t ldu, int taps, int C, T* __restrict__ state,
                  const int64_t* __restrict__ state_slots, const int32_t* __restrict__ qo_indptr) {
  const int b = blockIdx.x;
  const int c = blockIdx.y * 256 + threadIdx.x;
  if (c >= C) return;
  const int q0 = qo_indptr[b], n = qo_indptr[b + 1] - q0;
  if (n <= 0) return;
  T* st = state + state_slots[b] * (taps - 1) * C;
  for (int i = 0; i < taps - 1; ++i) {
    const int e = n - (taps - 1) + i;
    st[static_cast<int64_t>(i) * C + c] =
        e >= 0 ? u[static_cast<int64_t>(q0 + e) * ldu + c] : st[static_cast<int64_t>(taps - 1 + e) * C + c];
  }
}

template <typename T>
static int launch_conv(const void* u, int64_t ldu, const float* w, int taps, int C, const ConvOuts& outs, void* state,
                       const int64_t* slots, const int32_t* tok_req, const int32_t* qo, const int64_t* pos, int Tn, int n_req,
                       int one, cudaStream_t stream) {
  const T* up = static_cast<const T*>(u);
  T* st = static_cast<T*>(state);
  bool vec = C % 8 == 0 && ldu % 8 == 0 && aligned16(u) && aligned16(state) && aligned16(w) && taps >= 2 && taps <= 4;
  for (int i = 0; i < outs.n; ++i)
    vec = vec && outs.o[i].c0 % 8 == 0 && outs.o[i].c % 8 == 0 && outs.o[i].ldo % 8 == 0 && aligned16(outs.o[i].out);
  if (vec) {
    auto go = [&](auto one_kern, auto run_kern) -> int {
      const dim3 g(one ? Tn : ceil_div(Tn, kConvRun), ceil_div(C, 1024));
      return launch_kernel(one ? one_kern : run_kern, g, 128, 0, stream, Tn <= kPdlRows, up, ldu, w, C, outs, st, slots, tok_req,
                           qo, pos, Tn);
    };
    int r = FR_OK;
    if (taps == 2) r = go(&conv_vec_kernel<T, 2, true>, &conv_vec_kernel<T, 2, false>);
    if (taps == 3) r = go(&conv_vec_kernel<T, 3, true>, &conv_vec_kernel<T, 3, false>);
    if (taps == 4) r = go(&conv_vec_kernel<T, 4, true>, &conv_vec_kernel<T, 4, false>);
    if (r != FR_OK || one) return r;
    conv_state_kernel<T><<<dim3(n_req, ceil_div(C, 256)), 256, 0, stream>>>(up, ldu, taps, C, st, slots, qo);
    return launch_status();
  }
  dim3 grid(Tn, ceil_div(C, 256));
  if (one) {
    short_conv_kernel<T, true><<<grid, 256, 0, stream>>>(up, ldu, w, taps, C, outs, st, slots, tok_req, qo, pos);
    return launch_status();
  }
  short_conv_kernel<T, false><<<grid, 256, 0, stream>>>(up, ldu, w, taps, C, outs, st, slots, tok_req, qo, pos);
  if (launch_status() != FR_OK) return FR_ERR_CUDA;
  if (taps > 1) conv_state_kernel<T><<<dim3(n_req, ceil_div(C, 256)), 256, 0, stream>>>(up, ldu, taps, C, st, slots, qo);
  return launch_status();
}

template <typename T>
static int launch_norm(float* x, int64_t ldx, const float* weight, float offset, float eps, const float* partials,
                       int n_partials, int64_t ps, const int64_t* row_idx, void* out, int64_t ldo, int M, int W,
                       cudaStream_t stream) {
  const bool vec = W % 4 == 0 && W <= kNormThreads * 4 * kNormVec && ldx % 4 == 0 && ldo % 4 == 0 && aligned16(x) &&
                   aligned16(weight) && aligned16(out) && (partials == nullptr || (aligned16(partials) && ps % 4 == 0));
  T* o = static_cast<T*>(out);
  return launch_kernel(vec ? norm_kernel<T, true> : norm_kernel<T, false>, M, kNormThreads, 0, stream, M <= kPdlRows, x, ldx,
                       weight, offset, eps, partials, n_partials, ps, row_idx, o, ldo, W);
}

// ---------------------------------------------------------------------------
// x += partials, += coef * rms(y) * w per part, += a vector; then the norm of the result (or the result itself)
// ---------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ float4 ld4(const T* p);
template <>
__device__ __forceinline__ float4 ld4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <>
__device__ __forceinline__ float4 ld4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16lo(q.x), bf16hi(q.x), bf16lo(q.y), bf16hi(q.y));
}
template <typename T>
__device__ __forceinline__ void st4(T* p, const float4& v) {
  if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
  } else {
    *reinterpret_cast<float4*>(p) = v;
  }
}
__device__ __forceinline__ float sq4(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// Sum of a value over a CTA of NT threads (every thread gets it); `sums` is scratch that the next call may reuse only
// after another barrier, so callers alternate between two.
template <int NT>
__device__ __forceinline__ float cta_sum(float v, float* sums) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) sums[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) tot += sums[i];
  return tot;
}

// 1 / sqrt(mean + eps); the 16-bit results leave through the hardware's reciprocal root
template <typename T>
__device__ __forceinline__ float inv_rms(float sum, float inv_n, int n, float eps) {
  return sizeof(T) == 2 ? rsqrtf(fmaf(sum, inv_n, eps)) : 1.0f / sqrtf(sum / static_cast<float>(n) + eps);
}

// NT threads with NV float4 values each; NV 0: any width, re-reading what does not fit into registers. NP: parts at most;
// SHARES: they may come as shares of a split product
template <typename T, int NT, int NV, int NP, bool SHARES>
__global__ void __launch_bounds__(NT)
update_norm_kernel(const __grid_constant__ fr_norm_update u, int W) {
  __shared__ float sums[3][NT / 32];
  const float inv_w = 1.0f / static_cast<float>(W);
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t t = blockIdx.x;
  const int64_t src = u.row_idx != nullptr ? u.row_idx[t] : t;
  float* xr = u.x + src * u.ldx;
  T* o = static_cast<T*>(u.out) + t * u.ldo;
  const float* pr = u.n_partials > 0 ? u.partials + src * W : nullptr;
  const bool write_x = u.row_idx == nullptr && (pr != nullptr || u.n_parts > 0 || u.add != nullptr);
  if constexpr (NV > 0) {
    constexpr int kP = NP > 0 ? NP : 1;
    float4 v[NV], y[kP][NV];
    float ss[kP] = {};
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + threadIdx.x) * 4;
      v[i] = make_float4(0, 0, 0, 0);
#pragma unroll
      for (int p = 0; p < NP; ++p) y[p][i] = v[i];
      if (c >= W) continue;
      v[i] = *reinterpret_cast<const float4*>(xr + c);
#pragma unroll
      for (int p = 0; p < NP; ++p)
        if (p < u.n_parts) {
          if (!SHARES || u.parts[p].n_splits == 0) {
            y[p][i] = ld4<T>(static_cast<const T*>(u.parts[p].y) + src * u.parts[p].ldy + c);
          } else {
            for (int s = 0; s < u.parts[p].n_splits; ++s) {
              const float4 q = *reinterpret_cast<const float4*>(static_cast<const float*>(u.parts[p].y) + s * u.parts[p].ldy + src * W + c);
              y[p][i].x += q.x; y[p][i].y += q.y; y[p][i].z += q.z; y[p][i].w += q.w;
            }
          }
          ss[p] += sq4(y[p][i]);
        }
      if (pr != nullptr)
        for (int s = 0; s < u.n_partials; ++s) {
          const float4 q = *reinterpret_cast<const float4*>(pr + s * u.partial_stride + c);
          v[i].x += q.x; v[i].y += q.y; v[i].z += q.z; v[i].w += q.w;
        }
    }
    float r[kP] = {};
#pragma unroll
    for (int p = 0; p < NP; ++p)
      if (p < u.n_parts)
        r[p] = u.parts[p].coef * inv_rms<T>(cta_sum<NT>(ss[p], sums[p]), inv_w, W, u.eps);
    float sx = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + threadIdx.x) * 4;
      if (c >= W) continue;
#pragma unroll
      for (int p = 0; p < NP; ++p)
        if (p < u.n_parts) {
          const float4 w = *reinterpret_cast<const float4*>(u.parts[p].weight + c);
          v[i].x += y[p][i].x * r[p] * w.x; v[i].y += y[p][i].y * r[p] * w.y;
          v[i].z += y[p][i].z * r[p] * w.z; v[i].w += y[p][i].w * r[p] * w.w;
        }
      if (u.add != nullptr) {
        const float4 a = *reinterpret_cast<const float4*>(u.add + c);
        v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
      }
      if (write_x) *reinterpret_cast<float4*>(xr + c) = v[i];
      sx += sq4(v[i]);
    }
    if (u.out == nullptr) return;
    float rx = 1.0f;
    if (u.weight != nullptr) rx = inv_rms<T>(cta_sum<NT>(sx, sums[2]), inv_w, W, u.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + threadIdx.x) * 4;
      if (c >= W) continue;
      float4 w = make_float4(1, 1, 1, 1);
      if (u.weight != nullptr) {
        w = *reinterpret_cast<const float4*>(u.weight + c);
        w.x += u.offset; w.y += u.offset; w.z += u.offset; w.w += u.offset;
      }
      st4(o + c, make_float4(v[i].x * rx * w.x, v[i].y * rx * w.y, v[i].z * rx * w.z, v[i].w * rx * w.w));
    }
  } else {
    float r[2] = {0.f, 0.f};
    auto part = [&](int p, int c) {
      const fr_norm_part& q = u.parts[p];
      if (q.n_splits == 0) return ld_f(static_cast<const T*>(q.y) + src * q.ldy + c);
      float f = 0.f;
      for (int s = 0; s < q.n_splits; ++s) f += static_cast<const float*>(q.y)[s * q.ldy + src * W + c];
      return f;
    };
    for (int p = 0; p < u.n_parts; ++p) {
      float ss = 0.f;
      for (int c = threadIdx.x; c < W; c += NT) {
        const float f = part(p, c);
        ss += f * f;
      }
      r[p] = u.parts[p].coef * inv_rms<T>(cta_sum<NT>(ss, sums[p]), inv_w, W, u.eps);
    }
    auto value = [&](int c) {
      float f = xr[c];
      if (pr != nullptr)
        for (int s = 0; s < u.n_partials; ++s) f += pr[s * u.partial_stride + c];
      for (int p = 0; p < u.n_parts; ++p)
        f += part(p, c) * r[p] * u.parts[p].weight[c];
      if (u.add != nullptr) f += u.add[c];
      return f;
    };
    float rx = 1.0f;
    if (u.weight != nullptr && u.out != nullptr) {
      float sx = 0.f;
      for (int c = threadIdx.x; c < W; c += NT) {
        const float f = value(c);
        sx += f * f;
      }
      rx = inv_rms<T>(cta_sum<NT>(sx, sums[2]), inv_w, W, u.eps);
    }
    for (int c = threadIdx.x; c < W; c += NT) {  // a thread writes what only it reads
      const float f = value(c);
      if (write_x) xr[c] = f;
      if (u.out != nullptr) st_f(o + c, u.weight != nullptr ? f * rx * (u.offset + u.weight[c]) : f);
    }
  }
  if (u.out == nullptr) return;
  const int wpad = (W + 7) / 8 * 8;
  for (int c = W + threadIdx.x; c < wpad && c < u.ldo; c += NT) st_f(o + c, 0.f);
}

template <typename T, int NP, bool SHARES>
static int launch_update_norm_vec(const fr_norm_update& u, int M, int W, cudaStream_t stream) {
  const bool pdl = M <= kPdlRows;
  if (W <= 512) return launch_kernel(update_norm_kernel<T, 128, 1, NP, SHARES>, M, 128, 0, stream, pdl, u, W);
  // few rows: latency; two parts: registers
  if ((pdl || NP > 0) && W <= 2048) return launch_kernel(update_norm_kernel<T, 256, 2, NP, SHARES>, M, 256, 0, stream, pdl, u, W);
  if (W <= 2048) return launch_kernel(update_norm_kernel<T, 128, 4, NP, SHARES>, M, 128, 0, stream, pdl, u, W);
  if (NP > 0 && W <= 4096) return launch_kernel(update_norm_kernel<T, 512, 2, NP, SHARES>, M, 512, 0, stream, pdl, u, W);
  if (W <= 4096) return launch_kernel(update_norm_kernel<T, 256, 4, NP, SHARES>, M, 256, 0, stream, pdl, u, W);
  return launch_kernel(update_norm_kernel<T, 512, 4, NP, SHARES>, M, 512, 0, stream, pdl, u, W);
}

template <typename T>
static int launch_update_norm(const fr_norm_update& u, int M, int W, cudaStream_t stream) {
  bool vec = W % 4 == 0 && W <= 8192 && u.ldx % 4 == 0 && aligned16(u.x) && aligned16(u.weight) && aligned16(u.add) &&
             u.ldo % 4 == 0 && aligned16(u.out) && (u.n_partials == 0 || (aligned16(u.partials) && u.partial_stride % 4 == 0));
  bool shares = false;
  for (int p = 0; p < u.n_parts; ++p) {
    vec = vec && u.parts[p].ldy % 4 == 0 && aligned16(u.parts[p].y) && aligned16(u.parts[p].weight);
    shares = shares || u.parts[p].n_splits > 0;
  }
  if (vec && u.n_parts == 0) return launch_update_norm_vec<T, 0, false>(u, M, W, stream);
  if (vec) return shares ? launch_update_norm_vec<T, 2, true>(u, M, W, stream) : launch_update_norm_vec<T, 2, false>(u, M, W, stream);
  return launch_kernel(update_norm_kernel<T, kNormThreads, 0, 2, true>, M, kNormThreads, 0, stream, M <= kPdlRows, u, W);
}

// ---------------------------------------------------------------------------
// out = norm over groups of `size` columns, each by its own root mean square, with a silu gate before or after
// ---------------------------------------------------------------------------
constexpr int kGroupThreads = 256;

// NT threads per (row, group): a part of a warp, a warp or the CTA; eight columns at a time, NV of them per thread in
// registers
template <typename T, int NT, int NV>
__global__ void __launch_bounds__(kGroupThreads)
group_norm_kernel(const __grid_constant__ fr_group_norm a, int M) {
  __shared__ float sums[kGroupThreads / 32];
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t job = static_cast<int64_t>(blockIdx.x) * (kGroupThreads / NT) + threadIdx.x / NT;
  if (job - (threadIdx.x & 31) / NT >= static_cast<int64_t>(M) * a.groups) return;  // whole warps
  const bool live = job < static_cast<int64_t>(M) * a.groups;
  const int64_t t = live ? job / a.groups : 0;
  const int g = live ? static_cast<int>(job % a.groups) : 0, c0 = g * a.size, l = threadIdx.x % NT;
  const T* y = static_cast<const T*>(a.y) + t * a.ldy + c0;
  const T* z = a.gate_mode != FR_GATE_NONE ? static_cast<const T*>(a.gate) + t * a.ldg + c0 : nullptr;
  const float* w = a.weight + (a.weight_per_group ? c0 : 0);
  T* o = static_cast<T*>(a.out) + t * a.ldo + c0;
  float ss = 0.f;
  if constexpr (NV > 0) {
    float v[NV][8];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + l) * 8;
      if (c >= a.size) continue;
      raw_unpack(raw_load<T>(y + c), v[i]);
      if (a.gate_mode == FR_GATE_BEFORE) {
        float zv[8];
        raw_unpack(raw_load<T>(z + c), zv);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] *= silu_t<T>(zv[e]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[i][e], v[i][e], ss);
    }
    if constexpr (NT <= 32) {
#pragma unroll
      for (int o = NT / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    } else {
      ss = cta_sum<kGroupThreads>(ss, sums);
    }
    if (!live) return;
    const float r = 1.0f / sqrtf(ss / static_cast<float>(a.size) + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + l) * 8;
      if (c >= a.size) continue;
      float wv[8], f[8];
      *reinterpret_cast<float4*>(wv) = *reinterpret_cast<const float4*>(w + c);
      *reinterpret_cast<float4*>(wv + 4) = *reinterpret_cast<const float4*>(w + c + 4);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = v[i][e] * r * wv[e];
      if (a.gate_mode == FR_GATE_AFTER) {
        float zv[8];
        raw_unpack(raw_load<T>(z + c), zv);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= silu_t<T>(zv[e]);
      }
      conv_store8<T>(o + c, f);
    }
  } else {
    auto value = [&](int c) { return ld_f(y + c) * (a.gate_mode == FR_GATE_BEFORE ? silu_t<T>(ld_f(z + c)) : 1.0f); };
    for (int c = l; c < a.size; c += NT) {
      const float f = value(c);
      ss = fmaf(f, f, ss);
    }
    ss = NT == 32 ? warp_sum(ss) : cta_sum<kGroupThreads>(ss, sums);
    const float r = 1.0f / sqrtf(ss / static_cast<float>(a.size) + a.eps);
    for (int c = l; c < a.size; c += NT) {
      float f = value(c) * r * w[c];
      if (a.gate_mode == FR_GATE_AFTER) f *= silu_t<T>(ld_f(z + c));
      st_f(o + c, f);
    }
  }
  // columns up to the next multiple of eight: a matrix operand's padding
  const int n = a.groups * a.size, npad = (n + 7) / 8 * 8;
  if (g == a.groups - 1)
    for (int c = n + l; c < npad && c < a.ldo; c += NT) st_f(static_cast<T*>(a.out) + t * a.ldo + c, 0.f);
}

template <typename T>
static int launch_group_norm(const fr_group_norm& a, int M, cudaStream_t stream) {
  const bool vec = a.size % 8 == 0 && a.ldy % 8 == 0 && a.ldo % 8 == 0 && aligned16(a.y) && aligned16(a.out) && aligned16(a.weight) &&
                   (a.gate_mode == FR_GATE_NONE || (a.ldg % 8 == 0 && aligned16(a.gate)));
  const int64_t jobs = static_cast<int64_t>(M) * a.groups;
  const bool warp = a.size <= 1024;
  auto kern = warp ? group_norm_kernel<T, 32, 0> : group_norm_kernel<T, kGroupThreads, 0>;
  int per = kGroupThreads / 32;  // groups per CTA
  if (vec && warp) kern = a.size <= 256 ? group_norm_kernel<T, 32, 1> : group_norm_kernel<T, 32, 4>;
  if (vec && a.size <= 128) {
    kern = a.size <= 64 ? group_norm_kernel<T, 8, 1> : group_norm_kernel<T, 16, 1>;
    per = kGroupThreads / (a.size <= 64 ? 8 : 16);
  }
  if (vec && !warp && a.size <= kGroupThreads * 32)
    kern = a.size <= kGroupThreads * 16 ? group_norm_kernel<T, kGroupThreads, 2> : group_norm_kernel<T, kGroupThreads, 4>;
  return launch_kernel(kern, ceil_div(jobs, warp ? per : 1), kGroupThreads, 0, stream, M <= kPdlRows, a, M);
}

// ---------------------------------------------------------------------------
// queries and keys of one token: RMS norm over all heads at once, rotation, keys into the cache
// ---------------------------------------------------------------------------
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
  *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
  *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
}

__global__ void __launch_bounds__(256)
rotary_table_kernel(const float* __restrict__ inv_freq, int pairs, const int64_t* __restrict__ pos, float* __restrict__ table, int M) {
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t e = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (e >= static_cast<int64_t>(M) * pairs) return;
  const int64_t t = e / pairs;
  const int i = static_cast<int>(e % pairs);
  // the angle as a sum of two floats: its rounding alone would show at far positions
  const float p = static_cast<float>(pos[t]);
  const float2 f = reinterpret_cast<const float2*>(inv_freq)[i];
  const float hi = p * f.x, lo = fmaf(p, f.y, fmaf(p, f.x, -hi));
  float s, c;
  sincosf(hi, &s, &c);
  const float c1 = 1.0f - 0.5f * lo * lo, s1 = lo - lo * lo * lo * (1.0f / 6.0f);  // lo is at most half a place of hi
  table[t * 2 * pairs + i] = c * c1 - s * s1;
  table[t * 2 * pairs + pairs + i] = s * c1 + c * s1;
}

// A thread owns sixteen columns of one head, eight that turn with the other eight (or sixteen that do not), keeps their
// weights in registers and walks kRopeTokens tokens. rot_dims is a multiple of 16.
constexpr int kRopeTokens = 8;
template <typename T>
__global__ void __launch_bounds__(1024)
qk_norm_rope_units_kernel(const __grid_constant__ fr_qk_rope a, int M, int n_tokens) {
  __shared__ float sums[2][2][32];
  const int per_head = a.dim / 16, n_q = a.heads * per_head, n_units = (a.heads + a.kv_heads) * per_head;
  const int half = a.rot_dims / 2, tid = threadIdx.x, warp = tid >> 5, warps = blockDim.x >> 5;
  const bool live = tid < n_units, is_q = tid < n_q;
  const int u = live ? (is_q ? tid : tid - n_q) : 0, head = u / per_head, x = u % per_head;
  const bool turns = x < half / 8;
  const int c0 = turns ? x * 8 : a.rot_dims + (x - half / 8) * 16, c1 = turns ? half + x * 8 : c0 + 8;
  float w0[8], w1[8];
  const float* w = (is_q ? a.q_weight : a.k_weight) + head * a.dim;
  ld8(w + c0, w0);
  ld8(w + c1, w1);
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t t0 = static_cast<int64_t>(blockIdx.x) * n_tokens, t1 = t0 + n_tokens < M ? t0 + n_tokens : M;
  T* q = static_cast<T*>(a.q) + head * a.dim;
  const T* k = static_cast<const T*>(a.k) + head * a.dim;
  T* kc = static_cast<T*>(a.k_cache) + head * a.dim;
  // which sums a warp adds to, and what reads them: first and last unit of the warp
  const bool any_q = warp * 32 < n_q, any_k = warp * 32 + 31 >= n_q;
  const float inv_nq = 1.0f / static_cast<float>(a.heads * a.dim_true), inv_nk = 1.0f / static_cast<float>(a.kv_heads * a.dim_true);
  Raw8<T> r0 = raw_zero<T>(), r1 = r0;
  auto fetch = [&](int64_t t) {
    if (!live) return;
    const T* src = is_q ? q + t * a.ldq : k + t * a.ldk;
    r0 = raw_load<T>(src + c0);
    r1 = raw_load<T>(src + c1);
  };
  fetch(t0);
  for (int64_t t = t0; t < t1; ++t) {
    float v0[8], v1[8];
    raw_unpack(r0, v0);
    raw_unpack(r1, v1);
    if (t + 1 < t1) fetch(t + 1);
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(v0[e], v0[e], fmaf(v1[e], v1[e], ss));
    float (&s)[2][32] = sums[t & 1];
    if (any_q) {
      const float z = warp_sum(live && is_q ? ss : 0.f);
      if ((tid & 31) == 0) s[0][warp] = z;
    }
    if (any_k) {
      const float z = warp_sum(live && !is_q ? ss : 0.f);
      if ((tid & 31) == 0) s[1][warp] = z;
    }
    float cs[8], sn[8];
    if (live && turns) {
      ld8(a.table + t * a.rot_dims + c0, cs);
      ld8(a.table + t * a.rot_dims + half + c0, sn);
    }
    __syncthreads();
    if (!live) continue;
    float tot = 0.f;
    if (is_q)
      for (int i = 0; i * 32 < n_q; ++i) tot += s[0][i];
    else
      for (int i = n_q / 32; i < warps; ++i) tot += s[1][i];
    const float rr = inv_rms<T>(tot, is_q ? inv_nq : inv_nk, (is_q ? a.heads : a.kv_heads) * a.dim_true, a.eps);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float y0 = v0[e] * rr * w0[e], y1 = v1[e] * rr * w1[e];
      v0[e] = turns ? y0 * cs[e] - y1 * sn[e] : y0;
      v1[e] = turns ? y1 * cs[e] + y0 * sn[e] : y1;
    }
    T* dst = is_q ? q + t * a.ldq : kc + a.loc[t] * a.ldkc;
    conv_store8<T>(dst + c0, v0);
    conv_store8<T>(dst + c1, v1);
  }
}

// Any rotation: one token per CTA, eight columns per thread and turn.
constexpr int kRopeThreads = 1024;
template <typename T>
__global__ void __launch_bounds__(kRopeThreads)
qk_norm_rope_kernel(const __grid_constant__ fr_qk_rope a) {
  extern __shared__ float sm[];
  __shared__ float sums[2][kRopeThreads / 32];
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, half = a.rot_dims / 2, nt = blockDim.x;
  float* s_k = sm + nq;
  float* s_cos = s_k + nk;
  float* s_sin = s_cos + half;
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int64_t t = blockIdx.x;
  const int64_t slot = a.loc[t];
  T* q = static_cast<T*>(a.q) + t * a.ldq;
  const T* k = static_cast<const T*>(a.k) + t * a.ldk;
  float v[8], sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * 8; c < nq + nk; c += nt * 8) {
    raw_unpack(raw_load<T>(c < nq ? q + c : k + (c - nq)), v);
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    if (c < nq) sq += ss; else sk += ss;
    *reinterpret_cast<float4*>(sm + c) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(sm + c + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
  for (int i = threadIdx.x; i < a.rot_dims; i += nt) s_cos[i] = a.table[t * a.rot_dims + i];  // the sines follow
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    sums[0][threadIdx.x >> 5] = sq;
    sums[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();
  T* kc = static_cast<T*>(a.k_cache) + slot * a.ldkc;
  for (int c = threadIdx.x * 8; c < nq + nk; c += nt * 8) {
    const bool is_q = c < nq;
    const float* src = is_q ? sm : s_k;
    const float* w = is_q ? a.q_weight : a.k_weight;
    const int b = is_q ? c : c - nq, d0 = b % a.dim;
    float tot = 0.f;
    for (int i = 0; i < nt / 32; ++i) tot += sums[is_q ? 0 : 1][i];
    const float rr = 1.0f / sqrtf(tot / static_cast<float>((is_q ? a.heads : a.kv_heads) * a.dim_true) + a.eps);
    if (nt * 8 < nq + nk) ld8(sm + c, v);  // else the values of the one turn are still here
    float w8[8];
    ld8(w + b, w8);
    if (d0 >= a.rot_dims || half % 8 == 0) {  // eight dimensions turn with eight others, or none does
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= rr * w8[e];
      if (d0 < a.rot_dims) {
        const bool low = d0 < half;
        const int pair = low ? d0 : d0 - half, other = low ? b + half : b - half;
        float i8[8], c8[8], s8[8];
        ld8(src + other, i8);
        ld8(w + other, w8);
        ld8(s_cos + pair, c8);
        ld8(s_sin + pair, s8);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float it = i8[e] * rr * w8[e];
          v[e] = low ? v[e] * c8[e] - it * s8[e] : v[e] * c8[e] + it * s8[e];
        }
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int d = d0 + e;
        const float me = v[e] * rr * w8[e];
        v[e] = me;
        if (d < a.rot_dims) {
          const int pair = d < half ? d : d - half, other = d < half ? b + e + half : b + e - half;
          const float it = src[other] * rr * w[other];
          v[e] = d < half ? me * s_cos[pair] - it * s_sin[pair] : me * s_cos[pair] + it * s_sin[pair];
        }
      }
    }
    conv_store8<T>(is_q ? q + b : kc + b, v);
  }
}

}  // namespace lm
}  // namespace fr

using namespace fr;

extern "C" int fr_lm_embed(int dtype, const void* table, int64_t ldt, const int64_t* ids, float* x, int64_t ldx, int M, int W,
                           int vocab, float scale, int32_t* req_to_token, int64_t table_stride, const int64_t* rows,
                           const int64_t* pos, const int64_t* loc, cudaStream_t stream) {
  FR_CHECK_ARG((dtype == 0 || dtype == 1) && M >= 0 && W > 0 && vocab > 0 && ldt >= W && ldx >= W);
  if (M == 0) return FR_OK;
  FR_CHECK_ARG(table && ids && x && (req_to_token == nullptr || (rows && pos && loc)));
  if (dtype == 0)
    lm::embed_kernel<__nv_bfloat16><<<M, 256, 0, stream>>>(static_cast<const __nv_bfloat16*>(table), ldt, ids, x, ldx, W, vocab,
                                                           scale, req_to_token, table_stride, rows, pos, loc);
  else
    lm::embed_kernel<float><<<M, 256, 0, stream>>>(static_cast<const float*>(table), ldt, ids, x, ldx, W, vocab, scale,
                                                   req_to_token, table_stride, rows, pos, loc);
  return launch_status();
}

extern "C" int fr_lm_norm(int dtype, float* x, int64_t ldx, const float* weight, float offset, float eps,
                          const float* partials, int n_partials, int64_t partial_stride, const int64_t* row_idx, void* out,
                          int64_t ldo, int M, int W, cudaStream_t stream) {
  FR_CHECK_ARG((dtype == 0 || dtype == 1) && M >= 0 && W > 0 && ldx >= W && ldo >= W);
  if (M == 0) return FR_OK;
  FR_CHECK_ARG(x && weight && out && (n_partials == 0 || partials));
  if (n_partials == 0) partials = nullptr;
  return dtype == 0 ? lm::launch_norm<__nv_bfloat16>(x, ldx, weight, offset, eps, partials, n_partials, partial_stride,
                                                     row_idx, out, ldo, M, W, stream)
                    : lm::launch_norm<float>(x, ldx, weight, offset, eps, partials, n_partials, partial_stride, row_idx, out,
                                             ldo, M, W, stream);
}

extern "C" int fr_short_conv(int dtype, const void* u, int64_t ldu, const float* w, const float* bias, int act, int taps, int C,
                             const fr_conv_out* outs, int n_outs, void* state, const int64_t* state_slots, const int32_t* tok_req,
                             const int32_t* qo_indptr, const int64_t* pos, int T, int n_req, int one_token,
                             cudaStream_t stream) {
  FR_CHECK_ARG((act == FR_CONV_LINEAR || act == FR_CONV_SILU));
  FR_CHECK_ARG((dtype == 0 || dtype == 1) && T >= 0 && n_req >= 0 && taps >= 1 && C > 0 && ldu >= C && n_outs > 0 && n_outs <= 4);
  if (T == 0 || n_req == 0) return FR_OK;
  FR_CHECK_ARG(u && w && outs && state && state_slots && tok_req && qo_indptr && pos && (!one_token || T == n_req));
  lm::ConvOuts co{};
  co.n = n_outs;
  co.bias = bias;
  co.act = act;
  for (int i = 0; i < n_outs; ++i) {
    FR_CHECK_ARG(outs[i].out && outs[i].c0 >= 0 && outs[i].c > 0 && outs[i].c0 + outs[i].c <= C);
    co.o[i] = outs[i];
  }
  return dtype == 0 ? lm::launch_conv<__nv_bfloat16>(u, ldu, w, taps, C, co, state, state_slots, tok_req, qo_indptr, pos, T,
                                                     n_req, one_token, stream)
                    : lm::launch_conv<float>(u, ldu, w, taps, C, co, state, state_slots, tok_req, qo_indptr, pos, T, n_req,
                                             one_token, stream);
}

extern "C" int fr_lm_update_norm(const fr_norm_update* u, int M, int W, cudaStream_t stream) {
  FR_CHECK_ARG(u && (u->dtype == 0 || u->dtype == 1) && M >= 0 && W > 0 && u->ldx >= W && u->n_parts >= 0 && u->n_parts <= 2);
  if (M == 0) return FR_OK;
  FR_CHECK_ARG(u->x && (u->out == nullptr || u->ldo >= W) && u->n_partials >= 0 && (u->n_partials == 0 || u->partials));
  for (int p = 0; p < u->n_parts; ++p)
    FR_CHECK_ARG(u->parts[p].y && u->parts[p].weight && u->parts[p].ldy >= W && u->parts[p].n_splits >= 0);
  return u->dtype == 0 ? lm::launch_update_norm<__nv_bfloat16>(*u, M, W, stream) : lm::launch_update_norm<float>(*u, M, W, stream);
}

extern "C" int fr_lm_group_norm(const fr_group_norm* a, int M, cudaStream_t stream) {
  FR_CHECK_ARG(a && (a->dtype == 0 || a->dtype == 1) && M >= 0 && a->groups > 0 && a->size > 0);
  if (M == 0) return FR_OK;
  const int64_t n = static_cast<int64_t>(a->groups) * a->size;
  FR_CHECK_ARG(a->y && a->out && a->weight && a->ldy >= n && a->ldo >= n);
  FR_CHECK_ARG(a->gate_mode >= FR_GATE_NONE && a->gate_mode <= FR_GATE_AFTER && (a->gate_mode == FR_GATE_NONE || (a->gate && a->ldg >= n)));
  return a->dtype == 0 ? lm::launch_group_norm<__nv_bfloat16>(*a, M, stream) : lm::launch_group_norm<float>(*a, M, stream);
}

extern "C" int fr_lm_rotary_table(const float* inv_freq, int pairs, const int64_t* pos, float* table, int M, cudaStream_t stream) {
  FR_CHECK_ARG(pairs >= 0 && M >= 0);
  if (M == 0 || pairs == 0) return FR_OK;
  FR_CHECK_ARG(inv_freq && pos && table && (reinterpret_cast<uintptr_t>(inv_freq) & 7u) == 0);
  return launch_kernel(lm::rotary_table_kernel, ceil_div(static_cast<int64_t>(M) * pairs, 256), 256, 0, stream, M <= kPdlRows, inv_freq,
                       pairs, pos, table, M);
}

extern "C" int fr_lm_qk_norm_rope(const fr_qk_rope* a, int M, cudaStream_t stream) {
  FR_CHECK_ARG(a && (a->dtype == 0 || a->dtype == 1) && M >= 0 && a->heads > 0 && a->kv_heads > 0 && a->dim > 0 && a->dim % 8 == 0);
  if (M == 0) return FR_OK;
  FR_CHECK_ARG(a->dim_true > 0 && a->dim_true <= a->dim && a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->dim_true);
  FR_CHECK_ARG(a->q && a->k && a->k_cache && a->q_weight && a->k_weight && a->loc && (a->rot_dims == 0 || a->table));
  FR_CHECK_ARG(aligned16(a->q) && aligned16(a->k) && aligned16(a->k_cache) && aligned16(a->q_weight) && aligned16(a->k_weight) && a->ldq % 8 == 0 && a->ldk % 8 == 0 && a->ldkc % 8 == 0);
  const int units = (a->heads + a->kv_heads) * a->dim / 16;
  if (a->dim % 16 == 0 && a->rot_dims % 16 == 0 && units <= 1024 && aligned16(a->table)) {
    const int n = M > 148 * 16 ? lm::kRopeTokens : 1, threads = (units + 31) / 32 * 32;  // a few rows: a CTA each
    auto kern = a->dtype == 0 ? lm::qk_norm_rope_units_kernel<__nv_bfloat16> : lm::qk_norm_rope_units_kernel<float>;
    return launch_kernel(kern, ceil_div(M, n), threads, 0, stream, M <= kPdlRows, *a, M, n);
  }
  const int smem = ((a->heads + a->kv_heads) * a->dim + a->rot_dims) * 4;
  FR_CHECK_SUPPORTED(smem <= 200 * 1024);
  const int vecs = (a->heads + a->kv_heads) * a->dim / 8, threads = vecs >= lm::kRopeThreads ? lm::kRopeThreads : (vecs + 31) / 32 * 32;
  static PerDeviceFlag f0, f1;
  if (a->dtype == 0) {
    if (ensure_dyn_smem(f0, lm::qk_norm_rope_kernel<__nv_bfloat16>, 200 * 1024) != FR_OK) return FR_ERR_CUDA;
    return launch_kernel(lm::qk_norm_rope_kernel<__nv_bfloat16>, M, threads, smem, stream, M <= kPdlRows, *a);
  }
  if (ensure_dyn_smem(f1, lm::qk_norm_rope_kernel<float>, 200 * 1024) != FR_OK) return FR_ERR_CUDA;
  return launch_kernel(lm::qk_norm_rope_kernel<float>, M, threads, smem, stream, M <= kPdlRows, *a);
}
