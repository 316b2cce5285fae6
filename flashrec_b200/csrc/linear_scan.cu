// Recurrences with a matrix state per head (fr_linear_scan in the header):
//
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t,
//
// with a decay per key channel (gated linear attention: a low-rank projection, a sigmoid and a root) or per head
// (state-space duality: a step size that also scales v, and a skip). Everything here is fp32; q, k, v and o have the
// model's type.
//
//   scan_rows_kernel   any sizes, either type, decode and prompts: a thread keeps 8 rows x 4 columns of S in
//                      registers and walks the request's tokens, which are staged in shared memory in blocks
//   linear_chunk.cu    bf16 prompts on tcgen05, a chunk of tokens at a time
#include "fr_common.cuh"
#include "linear_scan.cuh"
#include "sm100_ptx.cuh"

namespace fr {
namespace scan {

constexpr int kRows = 8;  // rows of S per thread
constexpr int kCols = 4;  // columns of S per thread

struct RowsPlan {
  int vb;       // columns of S per CTA
  int tb;       // tokens staged at a time
  int threads;
  int smem;
};

template <typename T, bool CHANNEL>
__global__ void __launch_bounds__(1024)
scan_rows_kernel(const __grid_constant__ fr_linear_scan a, const RowsPlan pl, int min_tokens, int max_tokens,
                 const int32_t* __restrict__ flags) {
  extern __shared__ __align__(16) float sm[];
  const int np = state_rows(a.dim), vp = state_cols(a.vdim);
  const int rg_n = np / kRows, cq_n = pl.vb / kCols;
  float* s_q = sm;                                     // [tb][np]
  float* s_k = s_q + pl.tb * np;                       // [tb][np]
  float* s_v = s_k + pl.tb * np;                       // [tb][vb]
  float* s_y = s_v + pl.tb * pl.vb;                    // [tb][row groups][vb] shares of the output
  float* s_a = s_y + pl.tb * rg_n * pl.vb;             // [tb][np] (CHANNEL) or [tb]
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * pl.vb, tid = threadIdx.x, nt = blockDim.x;
  const int q0 = a.qo_indptr[b], q1 = a.qo_indptr[b + 1];
  if (q0 >= q1 || q1 - q0 > max_tokens || q1 - q0 < min_tokens) return;
  if (flags != nullptr && flags[b * a.heads + h] == 0) return;
  const int kh = h / (a.heads / a.key_heads);
  const int cq = tid % cq_n, rg = tid / cq_n;
  const bool active = rg < rg_n;
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
  float* st = a.state + ((a.state_slots[b] * a.heads + h) * np + rg * kRows) * static_cast<int64_t>(vp) + c0 + cq * kCols;
  uint64_t s2[kRows / 2][kCols];  // pairs of rows
#pragma unroll
  for (int r = 0; r < kRows / 2; ++r) {
    float4 lo = make_float4(0, 0, 0, 0), hi = lo;
    if (active && a.pos[q0] > 0) {
      lo = *reinterpret_cast<const float4*>(st + static_cast<int64_t>(2 * r) * vp);
      hi = *reinterpret_cast<const float4*>(st + static_cast<int64_t>(2 * r + 1) * vp);
    }
    s2[r][0] = pack2(lo.x, hi.x); s2[r][1] = pack2(lo.y, hi.y);
    s2[r][2] = pack2(lo.z, hi.z); s2[r][3] = pack2(lo.w, hi.w);
  }
  const T* qp = static_cast<const T*>(a.q);
  const T* kp = static_cast<const T*>(a.k);
  const T* vpt = static_cast<const T*>(a.v);
  for (int t0 = q0; t0 < q1; t0 += pl.tb) {
    const int n = min(pl.tb, q1 - t0);
    for (int e = tid; e < n * np; e += nt) {
      const int tt = e / np, c = e % np;
      const int64_t t = t0 + tt;
      const bool in = c < a.dim;
      s_q[e] = in ? to_f(qp[t * a.ldq + kh * a.dim + c]) * a.scale : 0.f;
      s_k[e] = in ? to_f(kp[t * a.ldk + kh * a.dim + c]) : 0.f;
      if constexpr (CHANNEL) s_a[e] = in ? expf(channel_log_decay(a, t, h * a.dim + c)) : 0.f;
    }
    for (int e = tid; e < n * pl.vb; e += nt) {
      const int tt = e / pl.vb, c = c0 + e % pl.vb;
      const int64_t t = t0 + tt;
      float v = c < a.vdim ? to_f(vpt[t * a.ldv + h * a.vdim + c]) : 0.f;
      if constexpr (!CHANNEL) v *= head_step(a, t, h);
      s_v[e] = v;
    }
    if constexpr (!CHANNEL)
      for (int tt = tid; tt < n; tt += nt) s_a[tt] = expf(-a.rate[h] * head_step(a, t0 + tt, h));
    __syncthreads();
    if (active) {
      for (int tt = 0; tt < n; ++tt) {
        const ulonglong2* kr = reinterpret_cast<const ulonglong2*>(s_k + tt * np + rg * kRows);
        const ulonglong2* qr = reinterpret_cast<const ulonglong2*>(s_q + tt * np + rg * kRows);
        const ulonglong2 ka = kr[0], kb = kr[1], qa = qr[0], qb = qr[1];
        const uint64_t k2[4] = {ka.x, ka.y, kb.x, kb.y}, qq[4] = {qa.x, qa.y, qb.x, qb.y};
        uint64_t a2[4];
        if constexpr (CHANNEL) {
          const ulonglong2* ar = reinterpret_cast<const ulonglong2*>(s_a + tt * np + rg * kRows);
          const ulonglong2 aa = ar[0], ab = ar[1];
          a2[0] = aa.x; a2[1] = aa.y; a2[2] = ab.x; a2[3] = ab.y;
        } else {
          a2[0] = a2[1] = a2[2] = a2[3] = dup2(s_a[tt]);
        }
        const float4 v = *reinterpret_cast<const float4*>(s_v + tt * pl.vb + cq * kCols);
        const uint64_t v2[4] = {dup2(v.x), dup2(v.y), dup2(v.z), dup2(v.w)};
        uint64_t y2[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
        for (int r = 0; r < kRows / 2; ++r)
#pragma unroll
          for (int c = 0; c < kCols; ++c) {
            s2[r][c] = fma2(a2[r], s2[r][c], mul2(k2[r], v2[c]));
            y2[c] = fma2(qq[r], s2[r][c], y2[c]);
          }
        float y[4];
#pragma unroll
        for (int c = 0; c < kCols; ++c) {
          float lo, hi;
          unpack2(y2[c], lo, hi);
          y[c] = lo + hi;
        }
        *reinterpret_cast<float4*>(s_y + (tt * rg_n + rg) * pl.vb + cq * kCols) = make_float4(y[0], y[1], y[2], y[3]);
      }
    }
    __syncthreads();
    for (int e = tid; e < n * pl.vb; e += nt) {
      const int tt = e / pl.vb, cc = e % pl.vb, c = c0 + cc;
      if (c >= a.vdim) continue;
      const int64_t t = t0 + tt;
      float y = 0.f;
      for (int g = 0; g < rg_n; ++g) y += s_y[(tt * rg_n + g) * pl.vb + cc];
      if (a.skip != nullptr) y = fmaf(skip, to_f(vpt[t * a.ldv + h * a.vdim + c]), y);
      from_f(static_cast<T*>(a.out) + t * a.ldo + h * a.vdim + c, y);
    }
  }
  if (!active) return;
#pragma unroll
  for (int r = 0; r < kRows / 2; ++r) {
    float4 lo, hi;
    unpack2(s2[r][0], lo.x, hi.x); unpack2(s2[r][1], lo.y, hi.y);
    unpack2(s2[r][2], lo.z, hi.z); unpack2(s2[r][3], lo.w, hi.w);
    *reinterpret_cast<float4*>(st + static_cast<int64_t>(2 * r) * vp) = lo;
    *reinterpret_cast<float4*>(st + static_cast<int64_t>(2 * r + 1) * vp) = hi;
  }
}

static bool plan_rows(const fr_linear_scan& a, int max_tokens, RowsPlan* pl) {
  const int np = state_rows(a.dim), vp = state_cols(a.vdim);
  pl->vb = vp % 32 == 0 ? 32 : 16;
  int threads = np / kRows * (pl->vb / kCols);
  if (threads > 1024) {
    pl->vb = 16;
    threads = np / kRows * (pl->vb / kCols);
  }
  if (threads > 1024) return false;
  pl->threads = (threads + 31) / 32 * 32;
  const bool channel = a.decay == FR_DECAY_CHANNEL;
  for (pl->tb = 16;; pl->tb /= 2) {
    pl->smem = pl->tb * (2 * np + pl->vb + np / kRows * pl->vb + (channel ? np : 1)) * 4 + 16;
    if (pl->smem <= 100 * 1024 && (pl->tb == 1 || pl->tb / 2 < max_tokens)) return true;
    if (pl->tb == 1) return pl->smem <= 200 * 1024;
  }
}

template <typename T, bool CHANNEL>
static int launch_rows(const fr_linear_scan& a, int n_req, int min_tokens, int max_tokens, const int32_t* flags, bool pdl,
                       cudaStream_t stream) {
  RowsPlan pl;
  FR_CHECK_SUPPORTED(plan_rows(a, max_tokens, &pl));
  static PerDeviceFlag f;
  if (ensure_dyn_smem(f, scan_rows_kernel<T, CHANNEL>, 200 * 1024) != FR_OK) return FR_ERR_CUDA;
  return launch_kernel(scan_rows_kernel<T, CHANNEL>, dim3(state_cols(a.vdim) / pl.vb, a.heads, n_req), pl.threads, pl.smem, stream, pdl,
                       a, pl, min_tokens, max_tokens, flags);
}

int rows_flagged(const fr_linear_scan& a, int n_req, int min_tokens, const int32_t* flags, cudaStream_t stream) {
  return launch_rows<__nv_bfloat16, true>(a, n_req, min_tokens, INT32_MAX, flags, false, stream);
}

}  // namespace scan
}  // namespace fr

using namespace fr;

extern "C" int64_t fr_linear_state_floats(int dim, int vdim) {
  return dim > 0 && vdim > 0 ? static_cast<int64_t>(scan::state_rows(dim)) * scan::state_cols(vdim) : -1;
}

extern "C" int fr_linear_scan_rows(const fr_linear_scan* a, int n_req, int max_tokens, int n_tokens, cudaStream_t stream) {
  const int st = scan::check_args(a);
  if (st != FR_OK) return st;
  FR_CHECK_ARG(n_req >= 0 && n_req <= 65535 && max_tokens >= 0 && n_tokens >= 0);
  if (n_req == 0 || max_tokens == 0) return FR_OK;
  const bool pdl = n_tokens <= kPdlRows;
  if (a->decay == FR_DECAY_CHANNEL)
    return a->dtype == 0 ? scan::launch_rows<__nv_bfloat16, true>(*a, n_req, 1, max_tokens, nullptr, pdl, stream)
                         : scan::launch_rows<float, true>(*a, n_req, 1, max_tokens, nullptr, pdl, stream);
  return a->dtype == 0 ? scan::launch_rows<__nv_bfloat16, false>(*a, n_req, 1, max_tokens, nullptr, pdl, stream)
                       : scan::launch_rows<float, false>(*a, n_req, 1, max_tokens, nullptr, pdl, stream);
}
