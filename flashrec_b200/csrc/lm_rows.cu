// Row kernels of the 16/32-bit decoder layers: embedding lookup into the fp32 residual stream (with the slot
// table entry of every new token), RMS norm of the fp32 stream, and the short causal convolution with its state.
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
};

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
      float y[8] = {};
#pragma unroll
      for (int k = 0; k < TAPS; ++k) {
        float f[8];
        raw_unpack(k < P ? win[k < P ? k : 0] : v[x], f);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(wr[k][i], f[i], y[i]);
      }
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
  float y = 0.f;
  for (int back = taps - 1; back >= 0; --back)
    y = fmaf(wc[taps - 1 - back], conv_tap(u, ldu, st, C, taps, t, e, p, c, back), y);
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

extern "C" int fr_short_conv(int dtype, const void* u, int64_t ldu, const float* w, int taps, int C, const fr_conv_out* outs,
                             int n_outs, void* state, const int64_t* state_slots, const int32_t* tok_req,
                             const int32_t* qo_indptr, const int64_t* pos, int T, int n_req, int one_token,
                             cudaStream_t stream) {
  FR_CHECK_ARG((dtype == 0 || dtype == 1) && T >= 0 && n_req >= 0 && taps >= 1 && C > 0 && ldu >= C && n_outs > 0 && n_outs <= 4);
  if (T == 0 || n_req == 0) return FR_OK;
  FR_CHECK_ARG(u && w && outs && state && state_slots && tok_req && qo_indptr && pos && (!one_token || T == n_req));
  lm::ConvOuts co{};
  co.n = n_outs;
  for (int i = 0; i < n_outs; ++i) {
    FR_CHECK_ARG(outs[i].out && outs[i].c0 >= 0 && outs[i].c > 0 && outs[i].c0 + outs[i].c <= C);
    co.o[i] = outs[i];
  }
  return dtype == 0 ? lm::launch_conv<__nv_bfloat16>(u, ldu, w, taps, C, co, state, state_slots, tok_req, qo_indptr, pos, T,
                                                     n_req, one_token, stream)
                    : lm::launch_conv<float>(u, ldu, w, taps, C, co, state, state_slots, tok_req, qo_indptr, pos, T, n_req,
                                             one_token, stream);
}
