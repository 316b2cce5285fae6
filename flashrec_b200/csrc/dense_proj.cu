// Matrix products of the 16/32-bit decoder layers, each with its layer's elementwise work in the epilogue:
//
//   fr_dense_proj       every projection of the normalised input h as ONE product with the merged weight; the
//                       column ranges leave through their own epilogues (plain store, store into KV-cache
//                       slots, SwiGLU or clamped GLU of interleaved gate / up rows, sigmoid with bias, GELU
//                       times a looked-up row)
//   fr_dense_gated_add  x += g1 * (A1 W1^T) + g2 * (A2 W2^T) on the fp32 residual stream
//
// Three implementations behind each:
//   dense_tc_kernel    bf16, persistent and warp-specialised like gemm_fp8.cu: warp 0 = TMA producer (128-byte
//                      swizzle, 64 bf16 per row), warp 1 = tcgen05.mma issuer (kind::f16, M = 128, fp32
//                      accumulators in TMEM, two buffers), warps 2..9 = epilogue
//   dense_rows_kernel  M <= 8 (decode): a warp streams four weight rows against all M activations, so the
//                      weights cross HBM once; the warps of a CTA may split K
//   dense_simt_kernel  f32 with more rows: 64 x 64 tiles, plain fp32 FMAs
#include "fr_common.cuh"
#include "sm100_ptx.cuh"

namespace fr {

int* device_status_ptr();  // capi.cu

namespace dense {

constexpr int kMaxSegs = 12;
struct Segs {
  fr_out_segment s[kMaxSegs];
  int n;
};
struct Parts {
  fr_gated_part p[2];
  int n;
};

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// eight consecutive elements as fp32
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void unpack8(const uint4& a, float (&v)[8]) {
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
  unpack8(*reinterpret_cast<const uint4*>(p), v);
}

// z * sigmoid(z) and sigmoid(z); FAST: the bf16 epilogues, whose result is rounded to 8 bits
template <bool FAST>
__device__ __forceinline__ float sigmoid_f(float z) {
  return FAST ? __fdividef(1.0f, 1.0f + __expf(-z)) : 1.0f / (1.0f + expf(-z));
}
template <bool FAST>
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f<FAST>(z); }

// gelu with the tanh approximation: 0.5 z (1 + tanh(u)) = z sigmoid(2 u)
template <bool FAST>
__device__ __forceinline__ float gelu_tanh_f(float z) {
  constexpr float kRoot = 0.7978845608028654f;  // sqrt(2 / pi)
  return z * sigmoid_f<FAST>(2.0f * kRoot * (z + 0.044715f * z * z * z));
}

// Ranges whose weight rows come in [32 gate | 32 up] blocks, and the activation of a pair.
__host__ __device__ __forceinline__ bool paired(const fr_out_segment& s) {
  return s.kind == FR_SEG_SWIGLU || s.kind == FR_SEG_GLU_CLAMP;
}
template <bool FAST>
__device__ __forceinline__ float pair_act(const fr_out_segment& s, float g, float u) {
  if (s.kind == FR_SEG_SWIGLU) return silu_f<FAST>(g) * u;
  g = fminf(g, s.limit);
  u = fminf(fmaxf(u, -s.limit), s.limit);
  return g * sigmoid_f<FAST>(s.alpha * g) * (u + s.up_bias);
}

__device__ __forceinline__ int seg_of(const Segs& sg, int col) {
  int i = 0;
#pragma unroll 1
  while (i + 1 < sg.n && col >= sg.s[i + 1].n0) ++i;
  return i;
}

// One value of one column range (column index within the range, already combined for SWIGLU).
template <typename T, bool FAST>
__device__ __forceinline__ void seg_write(const fr_out_segment& s, int64_t row, int c, float z) {
  if (c >= s.n) return;
  const int64_t r = s.row_map != nullptr ? s.row_map[row] : row;
  if (s.kind == FR_SEG_STORE_F32) {
    static_cast<float*>(s.out)[r * s.ldo + c] = z;
    return;
  }
  if (s.kind == FR_SEG_SIGMOID) z = sigmoid_f<FAST>(z + (s.bias != nullptr ? s.bias[c] : 0.f));
  if (s.kind == FR_SEG_GELU_MUL)
    z = gelu_tanh_f<FAST>(z) * to_f<T>(static_cast<const T*>(s.mul)[(s.mul_map != nullptr ? s.mul_map[row] : row) * s.ld_mul + c]);
  static_cast<T*>(s.out)[r * s.ldo + c] = from_f<T>(z);
}

// ---------------------------------------------------------------------------
// M <= 8: a warp takes four weight rows; KS warps of the CTA share them along K
// ---------------------------------------------------------------------------
constexpr int kRowsThreads = 256;

// ROWS weight rows (pointers) against MB activation rows, this warp's chunks of 256 columns
template <typename T, int MB>
__device__ __forceinline__ void rows_dot(const T* __restrict__ a, int64_t lda, const T* const (&w)[4], int K, int kwarp,
                                         int ks, int M, float (&acc)[4][MB]) {
  const int lane = threadIdx.x & 31;
#pragma unroll 2
  for (int k = kwarp * 256 + lane * 8; k < K; k += ks * 256) {
    float wv[4][8];
    if constexpr (sizeof(T) == 2) {
      uint4 raw[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) raw[r] = __ldcs(reinterpret_cast<const uint4*>(w[r] + k));
#pragma unroll
      for (int r = 0; r < 4; ++r) unpack8(raw[r], wv[r]);
    } else {
#pragma unroll
      for (int r = 0; r < 4; ++r) load8(w[r] + k, wv[r]);
    }
#pragma unroll
    for (int m = 0; m < MB; ++m) {
      float av[8];
      load8(a + (m < M ? m : 0) * lda + k, av);
#pragma unroll
      for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[r][m] = fmaf(wv[r][i], av[i], acc[r][m]);
    }
  }
}

// Start four weight rows on their way into L2 (weights never change: this may run before griddepcontrol.wait, while
// the previous kernel is still working).
template <typename T>
__device__ __forceinline__ void prefetch_rows(const T* const (&w)[4], int K, int kwarp, int ks) {
  constexpr int kLine = 128 / sizeof(T);
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int r = 0; r < 4; ++r)
    for (int k = (kwarp * 32 + lane) * kLine; k < K; k += ks * 32 * kLine)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(w[r] + k));
}

template <typename T, int MB>
__global__ void __launch_bounds__(kRowsThreads)
dense_rows_proj_kernel(const T* __restrict__ a, int64_t lda, const T* __restrict__ w, int64_t ldw, int M, int N, int K,
                       const __grid_constant__ Segs sg, int ks) {
  constexpr bool kFast = sizeof(T) == 2;
  __shared__ float red[8][4 * MB];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups_per_cta = (kRowsThreads / 32) / ks;
  const int grp = blockIdx.x * groups_per_cta + warp / ks;  // group of four weight rows
  const int kwarp = warp % ks;
  const bool live = grp * 4 < N;
  int si = 0, c0 = 0;
  float acc[4][MB] = {};
  const T* wr[4] = {};
  if (live) {
    si = seg_of(sg, grp * 4);
    const fr_out_segment& s = sg.s[si];
    const int local = grp * 4 - s.n0;
    if (paired(s)) {  // two channels: rows {gate c, gate c + 1, up c, up c + 1}
      c0 = local / 2;
      const int64_t g = s.n0 + (c0 / 32) * 64 + c0 % 32;
      wr[0] = w + g * ldw;
      wr[1] = w + (g + 1) * ldw;
      wr[2] = w + (g + 32) * ldw;
      wr[3] = w + (g + 33) * ldw;
    } else {
      c0 = local;
#pragma unroll
      for (int r = 0; r < 4; ++r) wr[r] = w + static_cast<int64_t>(grp * 4 + r) * ldw;
    }
    prefetch_rows<T>(wr, K, kwarp, ks);
  }
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  if (live) rows_dot<T, MB>(a, lda, wr, K, kwarp, ks, M, acc);
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int m = 0; m < MB; ++m) {
      const float v = warp_sum(acc[r][m]);
      if (lane == 0) red[warp][r * MB + m] = v;
    }
  __syncthreads();
  if (!live || kwarp != 0) return;
  const fr_out_segment& s = sg.s[si];
  if (paired(s)) {
    if (lane < 2 * MB) {
      const int r = lane / MB, m = lane % MB;
      float g = 0.f, u = 0.f;
      for (int k = 0; k < ks; ++k) {
        g += red[warp + k][r * MB + m];
        u += red[warp + k][(r + 2) * MB + m];
      }
      if (m < M) seg_write<T, kFast>(s, m, c0 + r, pair_act<kFast>(s, g, u));
    }
  } else if (lane < 4 * MB) {
    const int r = lane / MB, m = lane % MB;
    float z = 0.f;
    for (int k = 0; k < ks; ++k) z += red[warp + k][r * MB + m];
    if (m < M) seg_write<T, kFast>(s, m, c0 + r, z);
  }
}

template <typename T, int MB>
__global__ void __launch_bounds__(kRowsThreads)
dense_rows_gated_kernel(const __grid_constant__ Parts pt, float* __restrict__ x, int64_t ldx, int M, int N, T* __restrict__ copy,
                        int64_t ldc, int ks) {
  __shared__ float red[8][2][4 * MB];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups_per_cta = (kRowsThreads / 32) / ks;
  const int grp = blockIdx.x * groups_per_cta + warp / ks;
  const int kwarp = warp % ks;
  const bool live = grp * 4 < N;
  auto weight_rows = [&](const fr_gated_part& part, const T* (&wr)[4]) {
#pragma unroll
    for (int r = 0; r < 4; ++r)
      wr[r] = static_cast<const T*>(part.w) + static_cast<int64_t>(min(grp * 4 + r, N - 1)) * part.ldw;
  };
  if (live) {
    for (int p = 0; p < pt.n; ++p) {
      const T* wr[4];
      weight_rows(pt.p[p], wr);
      prefetch_rows<T>(wr, pt.p[p].K, kwarp, ks);
    }
  }
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  for (int p = 0; p < pt.n; ++p) {
    const fr_gated_part& part = pt.p[p];
    float acc[4][MB] = {};
    if (live) {
      const T* wr[4];
      weight_rows(part, wr);
      rows_dot<T, MB>(static_cast<const T*>(part.a), part.lda, wr, part.K, kwarp, ks, M, acc);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int m = 0; m < MB; ++m) {
        const float v = warp_sum(acc[r][m]);
        if (lane == 0) red[warp][p][r * MB + m] = v;
      }
  }
  __syncthreads();
  if (!live || kwarp != 0 || lane >= 4 * MB) return;
  const int r = lane / MB, m = lane % MB, n = grp * 4 + r;
  if (copy != nullptr && m < M && n >= N - 8)  // the padding behind the last columns
    for (int c = N + (n - (N - 8)); c < (N + 7) / 8 * 8 && c < ldc; c += 8) copy[m * ldc + c] = from_f<T>(0.f);
  if (m >= M || n >= N) return;
  float v = x[m * ldx + n];
  for (int p = 0; p < pt.n; ++p) {
    float z = 0.f;
    for (int k = 0; k < ks; ++k) z += red[warp + k][p][r * MB + m];
    const T* g = static_cast<const T*>(pt.p[p].gate);
    v += (g != nullptr ? to_f<T>(g[m * pt.p[p].ldg + n]) : 1.0f) * z;
  }
  x[m * ldx + n] = v;
  if (copy != nullptr) copy[m * ldc + n] = from_f<T>(v);
}

// ---------------------------------------------------------------------------
// f32, more rows: 64 x 64 tiles, 256 threads, 4 x 4 outputs per thread. Columns of a thread: two in the
// first half of the tile and the two 32 further on, so that a SwiGLU pair meets in one thread.
// ---------------------------------------------------------------------------
constexpr int kSimtK = 16;

__device__ __forceinline__ void simt_tile(const float* __restrict__ a, int64_t lda, const float* __restrict__ w, int64_t ldw,
                                          int M, int N, int K, int m0, int n0, float (&as)[kSimtK][68],
                                          float (&ws)[kSimtK][68], float (&acc)[4][4]) {
  const int tid = threadIdx.x, lr = tid >> 2, lk = (tid & 3) * 4;
  const int tx = tid & 15, ty = tid >> 4;
  for (int k0 = 0; k0 < K; k0 += kSimtK) {
    float4 av = make_float4(0, 0, 0, 0), wv = av;
    if (k0 + lk < K) {  // K is a multiple of 8
      if (m0 + lr < M) av = *reinterpret_cast<const float4*>(a + (m0 + lr) * lda + k0 + lk);
      if (n0 + lr < N) wv = *reinterpret_cast<const float4*>(w + (n0 + lr) * ldw + k0 + lk);
    }
    __syncthreads();
    as[lk][lr] = av.x; as[lk + 1][lr] = av.y; as[lk + 2][lr] = av.z; as[lk + 3][lr] = av.w;
    ws[lk][lr] = wv.x; ws[lk + 1][lr] = wv.y; ws[lk + 2][lr] = wv.z; ws[lk + 3][lr] = wv.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSimtK; ++k) {
      float ar[4], wr[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) ar[i] = as[k][ty * 4 + i];
      wr[0] = ws[k][tx * 2]; wr[1] = ws[k][tx * 2 + 1];
      wr[2] = ws[k][32 + tx * 2]; wr[3] = ws[k][33 + tx * 2];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], wr[j], acc[i][j]);
    }
  }
}

__global__ void __launch_bounds__(256)
dense_simt_proj_kernel(const float* __restrict__ a, int64_t lda, const float* __restrict__ w, int64_t ldw, int M, int N, int K,
                       const __grid_constant__ Segs sg) {
  __shared__ float as[kSimtK][68], ws[kSimtK][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  float acc[4][4] = {};
  simt_tile(a, lda, w, ldw, M, N, K, m0, n0, as, ws, acc);
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  for (int half = 0; half < 2; ++half) {
    const int col0 = n0 + half * 32;  // a 32-column chunk lies in one range
    if (col0 >= N) break;
    const fr_out_segment& s = sg.s[seg_of(sg, col0)];
    if (paired(s)) {
      if (half == 1) continue;
      const int ch = (col0 - s.n0) / 2 + tx * 2;
      for (int i = 0; i < 4; ++i) {
        const int row = m0 + ty * 4 + i;
        if (row >= M) break;
        for (int j = 0; j < 2; ++j) seg_write<float, false>(s, row, ch + j, pair_act<false>(s, acc[i][j], acc[i][2 + j]));
      }
    } else {
      for (int i = 0; i < 4; ++i) {
        const int row = m0 + ty * 4 + i;
        if (row >= M) break;
        for (int j = 0; j < 2; ++j) seg_write<float, false>(s, row, col0 - s.n0 + tx * 2 + j, acc[i][half * 2 + j]);
      }
    }
  }
}

__global__ void __launch_bounds__(256)
dense_simt_gated_kernel(const __grid_constant__ Parts pt, float* __restrict__ x, int64_t ldx, int M, int N, float* __restrict__ copy,
                        int64_t ldc) {
  __shared__ float as[kSimtK][68], ws[kSimtK][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float sum[4][4] = {};
  for (int p = 0; p < pt.n; ++p) {
    const fr_gated_part& part = pt.p[p];
    float acc[4][4] = {};
    simt_tile(static_cast<const float*>(part.a), part.lda, static_cast<const float*>(part.w), part.ldw, M, N, part.K, m0, n0,
              as, ws, acc);
    const float* g = static_cast<const float*>(part.gate);
    for (int i = 0; i < 4; ++i)
      for (int j = 0; j < 4; ++j) {
        const int row = m0 + ty * 4 + i, col = n0 + (j >> 1) * 32 + tx * 2 + (j & 1);
        if (row < M && col < N) sum[i][j] += (g != nullptr ? g[row * part.ldg + col] : 1.0f) * acc[i][j];
      }
  }
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 4; ++j) {
      const int row = m0 + ty * 4 + i, col = n0 + (j >> 1) * 32 + tx * 2 + (j & 1);
      if (row < M && col < N) {
        const float v = x[row * ldx + col] + sum[i][j];
        x[row * ldx + col] = v;
        if (copy != nullptr) copy[row * ldc + col] = v;
      } else if (copy != nullptr && row < M && col < (N + 7) / 8 * 8 && col < ldc) {
        copy[row * ldc + col] = 0.f;
      }
    }
}

// ---------------------------------------------------------------------------
// sum of the K shares of a split product, then the column ranges' epilogues
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
dense_finish_kernel(const float* __restrict__ partials, int n_splits, int M, int N, const __grid_constant__ Segs sg) {
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int row = blockIdx.y, col = blockIdx.x * 256 + threadIdx.x;
  if (col >= N) return;
  const fr_out_segment& s = sg.s[seg_of(sg, col)];
  auto sum = [&](int c) {
    float z = 0.f;
    for (int i = 0; i < n_splits; ++i) z += partials[(static_cast<int64_t>(i) * M + row) * N + c];
    return z;
  };
  const int local = col - s.n0;
  constexpr bool kFast = sizeof(T) == 2;
  if (!paired(s)) {
    seg_write<T, kFast>(s, row, local, sum(col));
  } else if (local % 64 < 32) {
    seg_write<T, kFast>(s, row, local / 64 * 32 + local % 64, pair_act<kFast>(s, sum(col), sum(col + 32)));
  }
}

// ---------------------------------------------------------------------------
// bf16 on tcgen05
// ---------------------------------------------------------------------------
constexpr int kBlockM = 128;
constexpr int kBlockK = 64;  // bf16 elements: one 128-byte swizzle span
constexpr int kUmmaK = 16;
constexpr int kEpiWarps = 8;
constexpr int kThreads = 64 + kEpiWarps * 32;
enum Epi { kEpiSegs = 0, kEpiAdd = 1, kEpiPartial = 2 };

template <int BLOCK_N>
struct Cfg {
  static constexpr int kStageA = kBlockM * kBlockK * 2;
  static constexpr int kStageB = BLOCK_N * kBlockK * 2;
  static constexpr int kStageBytes = kStageA + kStageB;
  static constexpr int kStages = BLOCK_N == 256 ? 4 : (BLOCK_N == 128 ? 6 : 8);
  static constexpr int kTmemCols = 2 * BLOCK_N;
  static constexpr int kBarBytes = (2 * kStages + 4) * 8 + 16;
  static constexpr int kSmemBytes = 1024 + kStages * kStageBytes + kBarBytes;
};

struct TcArgs {
  int M, N;
  int n_parts;
  int kb[2];         // k-blocks per part
  int splits[2];     // kEpiPartial: K splits per part
  Segs segs;         // kEpiSegs
  float* x;          // kEpiAdd
  int64_t ldx;
  const __nv_bfloat16* gate[2];
  int64_t ldg[2];
  float* partials;   // kEpiPartial: [splits, M, N]
  __nv_bfloat16* copy;  // kEpiAdd: the new x as bf16, or null
  int64_t ldc;
};

// Work of a CTA in order: kEpiSegs / kEpiAdd: tile after tile, the parts of a tile back to back (its second
// accumulator is added by the same threads as its first); kEpiPartial: one K share of one part of one tile.
struct Job {
  int mb, nb, part, kb0, kb1, slot;
};
template <int EPI>
__device__ __forceinline__ Job job_at(const TcArgs& g, int unit, int sub, int m_blocks, int n_blocks) {
  Job j;
  int tile = unit;
  j.part = sub;
  j.kb0 = 0;
  j.slot = 0;
  if (EPI == kEpiPartial) {
    const int per_tile = g.splits[0] + g.splits[1];
    tile = unit / per_tile;
    const int s = unit % per_tile;
    j.part = s < g.splits[0] ? 0 : 1;
    const int i = j.part == 0 ? s : s - g.splits[0];
    const int n = g.splits[j.part], kb = g.kb[j.part];
    j.kb0 = static_cast<int>(static_cast<int64_t>(kb) * i / n);
    j.kb1 = static_cast<int>(static_cast<int64_t>(kb) * (i + 1) / n);
    j.slot = s;
  } else {
    j.kb1 = g.kb[sub];
  }
  constexpr int kGroup = 8;  // row blocks per raster group: A streams once, the group's B blocks stay in L2
  const int per_group = kGroup * n_blocks;
  const int first = tile / per_group * kGroup;
  const int rows = min(kGroup, m_blocks - first);
  const int t = tile - tile / per_group * per_group;
  j.mb = first + t % rows;
  j.nb = t / rows;
  return j;
}

__device__ __forceinline__ void store32_bf16(__nv_bfloat16* dst, const float (&v)[32], int nvalid) {
  if (nvalid >= 32 && (reinterpret_cast<uintptr_t>(dst) & 15u) == 0) {
    uint32_t w[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) w[i] = pack_bf16(v[2 * i], v[2 * i + 1]);
    if ((reinterpret_cast<uintptr_t>(dst) & 31u) == 0) {
      const uint32_t w0[8] = {w[0], w[1], w[2], w[3], w[4], w[5], w[6], w[7]};
      const uint32_t w1[8] = {w[8], w[9], w[10], w[11], w[12], w[13], w[14], w[15]};
      ptx::st_global_v8(dst, w0);
      ptx::st_global_v8(dst + 16, w1);
    } else {
      uint4* d4 = reinterpret_cast<uint4*>(dst);
#pragma unroll
      for (int i = 0; i < 4; ++i) d4[i] = make_uint4(w[4 * i], w[4 * i + 1], w[4 * i + 2], w[4 * i + 3]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (i < nvalid) dst[i] = __float2bfloat16_rn(v[i]);
  }
}

// 32 fp32 values to / from consecutive addresses; vector accesses when the row allows them
__device__ __forceinline__ void store32_f32(float* dst, const float (&v)[32], int nvalid) {
  if (nvalid >= 32 && (reinterpret_cast<uintptr_t>(dst) & 15u) == 0) {
    float4* d4 = reinterpret_cast<float4*>(dst);
#pragma unroll
    for (int i = 0; i < 8; ++i) d4[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (i < nvalid) dst[i] = v[i];
  }
}

template <int BLOCK_N, int EPI>
__global__ void __launch_bounds__(kThreads, 1)
dense_tc_kernel(const __grid_constant__ CUtensorMap ta0, const __grid_constant__ CUtensorMap tb0,
                const __grid_constant__ CUtensorMap ta1, const __grid_constant__ CUtensorMap tb1,
                const __grid_constant__ TcArgs g, int* status) {
  using C = Cfg<BLOCK_N>;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::kStages * C::kStageBytes);
  const uint32_t bar_full = ptx::smem_u32(bars);
  const uint32_t bar_empty = bar_full + 8 * C::kStages;
  const uint32_t bar_tfull = bar_empty + 8 * C::kStages;
  const uint32_t bar_tempty = bar_tfull + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * C::kStages + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int m_blocks = (g.M + kBlockM - 1) / kBlockM;
  const int n_blocks = (g.N + BLOCK_N - 1) / BLOCK_N;
  const int subs = EPI == kEpiPartial ? 1 : g.n_parts;
  const int num_units = m_blocks * n_blocks * (EPI == kEpiPartial ? g.splits[0] + g.splits[1] : 1);

  if (threadIdx.x == 0) {
    for (int s = 0; s < C::kStages; ++s) {
      ptx::mbar_init(bar_full + 8 * s, 1);
      ptx::mbar_init(bar_empty + 8 * s, 1);
    }
    for (int b = 0; b < 2; ++b) {
      ptx::mbar_init(bar_tfull + 8 * b, 1);
      ptx::mbar_init(bar_tempty + 8 * b, kEpiWarps);
    }
    *abort_flag = 0;
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&ta0);
    ptx::prefetch_tmap(&tb0);
  }
  if (warp == 1) {
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), C::kTmemCols);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();

  if (warp == 0) {
    if (lane == 0) {
      uint32_t stage = 0, phase = 0;
      bool ok = true;
      for (int unit = blockIdx.x; unit < num_units && ok; unit += gridDim.x) {
        for (int sub = 0; sub < subs && ok; ++sub) {
          const Job j = job_at<EPI>(g, unit, sub, m_blocks, n_blocks);
          const CUtensorMap* ta = j.part == 0 ? &ta0 : &ta1;
          const CUtensorMap* tb = j.part == 0 ? &tb0 : &tb1;
          for (int kb = j.kb0; kb < j.kb1; ++kb) {
            ok = ptx::mbar_wait(bar_empty + 8 * stage, phase ^ 1u, abort_flag, status, 61);
            if (!ok) break;
            const uint32_t sa = base + stage * C::kStageBytes;
            ptx::mbar_expect_tx(bar_full + 8 * stage, C::kStageBytes);
            ptx::tma_load_2d(sa, ta, kb * kBlockK, j.mb * kBlockM, bar_full + 8 * stage);
            ptx::tma_load_2d(sa + C::kStageA, tb, kb * kBlockK, j.nb * BLOCK_N, bar_full + 8 * stage);
            if (++stage == C::kStages) { stage = 0; phase ^= 1u; }
          }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = ptx::make_idesc(1u, 1u, kBlockM, BLOCK_N);
      uint32_t stage = 0, phase = 0;
      bool ok = true;
      int it = 0;
      for (int unit = blockIdx.x; unit < num_units && ok; unit += gridDim.x) {
        for (int sub = 0; sub < subs && ok; ++sub, ++it) {
          const Job j = job_at<EPI>(g, unit, sub, m_blocks, n_blocks);
          const uint32_t buf = it & 1;
          ok = ptx::mbar_wait(bar_tempty + 8 * buf, ((it >> 1) & 1) ^ 1u, abort_flag, status, 62);
          if (!ok) break;
          ptx::tc_fence_after();
          const uint32_t d_tmem = tmem_base + buf * BLOCK_N;
          for (int kb = j.kb0; kb < j.kb1; ++kb) {
            ok = ptx::mbar_wait(bar_full + 8 * stage, phase, abort_flag, status, 63);
            if (!ok) break;
            ptx::tc_fence_after();
            const uint32_t sa = base + stage * C::kStageBytes;
            const uint64_t a_desc = ptx::smem_desc_sw128(sa);
            const uint64_t b_desc = ptx::smem_desc_sw128(sa + C::kStageA);
#pragma unroll
            for (int k = 0; k < kBlockK / kUmmaK; ++k)
              ptx::mma_f16(d_tmem, a_desc + 2u * k, b_desc + 2u * k, idesc, (kb > j.kb0 || k > 0) ? 1u : 0u);
            ptx::tc_commit(bar_empty + 8 * stage);
            if (++stage == C::kStages) { stage = 0; phase ^= 1u; }
          }
          if (ok) ptx::tc_commit(bar_tfull + 8 * buf);
        }
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3;
    const int part_of_cols = (warp - 2) >> 2;  // two warps per lane quadrant: even / odd chunks
    bool ok = true;
    int it = 0;
    for (int unit = blockIdx.x; unit < num_units && ok; unit += gridDim.x) {
      for (int sub = 0; sub < subs && ok; ++sub, ++it) {
        const Job j = job_at<EPI>(g, unit, sub, m_blocks, n_blocks);
        const uint32_t buf = it & 1;
        const int row = j.mb * kBlockM + quad * 32 + lane;
        const int n0 = j.nb * BLOCK_N;
        int okw = 0;
        if (lane == 0) okw = ptx::mbar_wait(bar_tfull + 8 * buf, (it >> 1) & 1, abort_flag, status, 64) ? 1 : 0;
        okw = __shfl_sync(0xffffffffu, okw, 0);
        if (!okw) { ok = false; break; }
        ptx::tc_fence_after();
        const uint32_t taddr = tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + buf * BLOCK_N;
        if constexpr (EPI == kEpiSegs) {
#pragma unroll 1
          for (int c = part_of_cols; c < BLOCK_N / 64; c += 2) {  // pairs of 32-column chunks
            const int col = n0 + c * 64;
            if (col >= g.N) break;
            uint32_t r0[32], r1[32];
            ptx::tmem_ld_32x32(taddr + c * 64, r0);
            ptx::tmem_ld_32x32(taddr + c * 64 + 32, r1);
            ptx::tmem_ld_wait();
            if (row < g.M) {
            const fr_out_segment& s0 = g.segs.s[seg_of(g.segs, col)];
            if (paired(s0)) {
              const int ch = (col - s0.n0) / 2;
              float v[32];
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = pair_act<true>(s0, __uint_as_float(r0[i]), __uint_as_float(r1[i]));
              const int64_t r = s0.row_map != nullptr ? s0.row_map[row] : row;
              store32_bf16(static_cast<__nv_bfloat16*>(s0.out) + r * s0.ldo + ch, v, s0.n - ch);
            } else {
#pragma unroll
              for (int half = 0; half < 2; ++half) {
                const int hc = col + half * 32;
                if (hc < g.N) {
                  const fr_out_segment& s = g.segs.s[seg_of(g.segs, hc)];
                  const int lc = hc - s.n0, nvalid = s.n - lc;
                  float v[32];
#pragma unroll
                  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(half == 0 ? r0[i] : r1[i]);
                  if (nvalid > 0) {
                    const int64_t r = s.row_map != nullptr ? s.row_map[row] : row;
                    if (s.kind == FR_SEG_STORE_F32) {
                      store32_f32(static_cast<float*>(s.out) + r * s.ldo + lc, v, nvalid);
                    } else {
                      if (s.kind == FR_SEG_SIGMOID) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) {
                          const float b = (s.bias != nullptr && i < nvalid) ? __ldg(s.bias + lc + i) : 0.f;
                          v[i] = sigmoid_f<true>(v[i] + b);
                        }
                      }
                      if (s.kind == FR_SEG_GELU_MUL) {
                        const __nv_bfloat16* mul = static_cast<const __nv_bfloat16*>(s.mul) +
                                                   (s.mul_map != nullptr ? s.mul_map[row] : row) * s.ld_mul + lc;
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                          if (i < nvalid) v[i] = gelu_tanh_f<true>(v[i]) * __bfloat162float(__ldg(mul + i));
                      }
                      store32_bf16(static_cast<__nv_bfloat16*>(s.out) + r * s.ldo + lc, v, nvalid);
                    }
                  }
                }
              }
            }
            }
            __syncwarp();  // the next tcgen05.ld is a whole-warp instruction
          }
        } else {
#pragma unroll 1
          for (int c = part_of_cols; c < BLOCK_N / 32; c += 2) {
            const int col = n0 + c * 32;
            const int nvalid = g.N - col;
            if (nvalid <= 0) break;
            uint32_t r[32];
            ptx::tmem_ld_32x32(taddr + c * 32, r);
            // the operands of the update are in flight while the accumulator is read
            const __nv_bfloat16* gp = g.gate[j.part];
            float gt[32];
            const bool live = row < g.M;
            const __nv_bfloat16* gr = gp + (live ? row : 0) * g.ldg[j.part] + col;
            if (gp != nullptr && nvalid >= 32 && (reinterpret_cast<uintptr_t>(gr) & 15u) == 0) {
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                float t[8];
                unpack8(__ldg(reinterpret_cast<const uint4*>(gr) + i), t);
#pragma unroll
                for (int e = 0; e < 8; ++e) gt[i * 8 + e] = t[e];
              }
            } else {
#pragma unroll
              for (int i = 0; i < 32; ++i) gt[i] = gp == nullptr ? 1.0f : (i < nvalid ? __bfloat162float(gr[i]) : 0.f);
            }
            float v[32];
            if constexpr (EPI == kEpiAdd) {
              float* xr = g.x + (live ? row : 0) * g.ldx + col;
              if (nvalid >= 32 && (reinterpret_cast<uintptr_t>(xr) & 15u) == 0) {
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                  const float4 t = reinterpret_cast<const float4*>(xr)[i];
                  v[4 * i] = t.x; v[4 * i + 1] = t.y; v[4 * i + 2] = t.z; v[4 * i + 3] = t.w;
                }
              } else {
#pragma unroll
                for (int i = 0; i < 32; ++i) v[i] = i < nvalid ? xr[i] : 0.f;
              }
              ptx::tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = fmaf(gt[i], __uint_as_float(r[i]), v[i]);
              if (live) store32_f32(xr, v, nvalid);
              if (live && g.copy != nullptr && sub + 1 == subs) {
                __nv_bfloat16* cr = g.copy + row * g.ldc + col;
                store32_bf16(cr, v, nvalid);
                if (nvalid < 32)
                  for (int c = nvalid; (col + c) % 8 != 0 && col + c < g.ldc; ++c) cr[c] = __float2bfloat16_rn(0.f);
              }
            } else {
              ptx::tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = gt[i] * __uint_as_float(r[i]);
              if (live) store32_f32(g.partials + (static_cast<int64_t>(j.slot) * g.M + row) * g.N + col, v, nvalid);
            }
            __syncwarp();
          }
        }
        ptx::tc_fence_before();
        __syncwarp();
        if (lane == 0) ptx::mbar_arrive(bar_tempty + 8 * buf);
      }
    }
  }

  ptx::tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    ptx::tc_fence_after();
    ptx::tmem_dealloc(tmem_base, C::kTmemCols);
  }
}

// ---------------------------------------------------------------------------
// host side
// ---------------------------------------------------------------------------
typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiledFn encode_fn() {
  static EncodeTiledFn fn = []() -> EncodeTiledFn {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess) return nullptr;
    if (q != cudaDriverEntryPointSuccess) return nullptr;
    return reinterpret_cast<EncodeTiledFn>(ptr);
  }();
  return fn;
}

// bf16 [rows, cols] with a row pitch, box of 64 columns x box_rows, 128-byte swizzle, zero fill outside
int make_tmap_bf16_2d(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, int64_t pitch, uint32_t box_rows) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return FR_ERR_CUDA;
  cuuint64_t dims[2] = {cols, rows};
  cuuint64_t strides[1] = {static_cast<cuuint64_t>(pitch) * 2};
  cuuint32_t box[2] = {64, box_rows};
  cuuint32_t estr[2] = {1, 1};
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? FR_OK : FR_ERR_CUDA;
}

template <int BLOCK_N, int EPI>
static int launch_tc(const TcArgs& g, const fr_gated_part* parts, cudaStream_t stream) {
  CUtensorMap ta[2], tb[2];
  for (int p = 0; p < 2; ++p) {
    const fr_gated_part& q = parts[p < g.n_parts ? p : 0];
    int st = make_tmap_bf16_2d(&ta[p], q.a, q.K, g.M, q.lda, kBlockM);
    if (st == FR_OK) st = make_tmap_bf16_2d(&tb[p], q.w, q.K, g.N, q.ldw, BLOCK_N);
    if (st != FR_OK) return st;
  }
  auto kern = dense_tc_kernel<BLOCK_N, EPI>;
  static PerDeviceFlag attr_done;
  if (ensure_dyn_smem(attr_done, kern, Cfg<BLOCK_N>::kSmemBytes) != FR_OK) return FR_ERR_CUDA;
  int* status = device_status_ptr();
  if (!status) return FR_ERR_CUDA;
  const int64_t units = static_cast<int64_t>(ceil_div(g.M, kBlockM)) * ceil_div(g.N, BLOCK_N) *
                        (EPI == kEpiPartial ? g.splits[0] + g.splits[1] : 1);
  const int grid = static_cast<int>(units < device_sm_count() ? units : device_sm_count());
  return launch_kernel(kern, grid, kThreads, Cfg<BLOCK_N>::kSmemBytes, stream, g.M <= kPdlRows, ta[0], tb[0], ta[1], tb[1], g,
                       status);
}

// Tile width with the least work on the busiest SM: rounds of tiles times the rows of A and B that a tile brings in.
static int pick_block_n(int M, int N) {
  const int64_t sms = device_sm_count(), mb = ceil_div(M, kBlockM);
  int best = 0;
  int64_t best_cost = 0;
  for (int bn = 256; bn >= 64; bn /= 2) {
    const int64_t cost = (mb * ceil_div(N, bn) + sms - 1) / sms * (kBlockM + bn);
    if (best == 0 || cost < best_cost) {
      best = bn;
      best_cost = cost;
    }
  }
  return best;
}

static int rows_ks(int N, int K) {
  // warps per CTA that share a group of four rows along K: several waves of small CTAs, so that the last one is
  // short, as long as a warp keeps two steps of 256 columns
  const int64_t warps = ceil_div(N, 4);
  int ks = 1;
  while (ks < 8 && ((warps * ks < 148 * 16 && K / (ks * 2) >= 256) || (warps * ks < 148 * 96 && K / (ks * 2) >= 512))) ks *= 2;
  return ks;
}

template <typename T>
static int launch_rows_proj(const void* a, int64_t lda, const void* w, int64_t ldw, int M, int N, int K, const Segs& sg,
                            cudaStream_t stream) {
  const int ks = rows_ks(N, K);
  const int grid = ceil_div(ceil_div(N, 4), (kRowsThreads / 32) / ks);
  const T* A = static_cast<const T*>(a);
  const T* W = static_cast<const T*>(w);
  if (M == 1) return launch_kernel(dense_rows_proj_kernel<T, 1>, grid, kRowsThreads, 0, stream, true, A, lda, W, ldw, M, N, K, sg, ks);
  if (M == 2) return launch_kernel(dense_rows_proj_kernel<T, 2>, grid, kRowsThreads, 0, stream, true, A, lda, W, ldw, M, N, K, sg, ks);
  if (M <= 4) return launch_kernel(dense_rows_proj_kernel<T, 4>, grid, kRowsThreads, 0, stream, true, A, lda, W, ldw, M, N, K, sg, ks);
  return launch_kernel(dense_rows_proj_kernel<T, 8>, grid, kRowsThreads, 0, stream, true, A, lda, W, ldw, M, N, K, sg, ks);
}

template <typename T>
static int launch_rows_gated(const Parts& pt, float* x, int64_t ldx, int M, int N, void* copy_out, int64_t ldc, cudaStream_t stream) {
  T* copy = static_cast<T*>(copy_out);
  int K = 0;
  for (int p = 0; p < pt.n; ++p) K = K > pt.p[p].K ? K : pt.p[p].K;
  const int ks = rows_ks(N, K);
  const int grid = ceil_div(ceil_div(N, 4), (kRowsThreads / 32) / ks);
  if (M == 1) return launch_kernel(dense_rows_gated_kernel<T, 1>, grid, kRowsThreads, 0, stream, true, pt, x, ldx, M, N, copy, ldc, ks);
  if (M == 2) return launch_kernel(dense_rows_gated_kernel<T, 2>, grid, kRowsThreads, 0, stream, true, pt, x, ldx, M, N, copy, ldc, ks);
  if (M <= 4) return launch_kernel(dense_rows_gated_kernel<T, 4>, grid, kRowsThreads, 0, stream, true, pt, x, ldx, M, N, copy, ldc, ks);
  return launch_kernel(dense_rows_gated_kernel<T, 8>, grid, kRowsThreads, 0, stream, true, pt, x, ldx, M, N, copy, ldc, ks);
}

static bool operand_ok(const void* p, int64_t ld, int K) {
  return p != nullptr && (reinterpret_cast<uintptr_t>(p) & 15u) == 0 && ld % 8 == 0 && ld >= K && K % 8 == 0 && K > 0;
}

// K shares of the two parts for few-row products: about one work unit per SM in all.
static void plan_splits(int M, int N, int kb0, int kb1, int* s0, int* s1) {
  *s0 = *s1 = 0;
  const int64_t tiles = static_cast<int64_t>(ceil_div(M, kBlockM)) * ceil_div(N, 64);
  if (tiles * 2 > device_sm_count() || M > 1024) return;  // the tiles alone keep the SMs busy
  const int want = static_cast<int>(device_sm_count() / tiles);
  const int total = kb0 + kb1;
  int a = static_cast<int>((static_cast<int64_t>(want) * kb0 + total / 2) / total);
  a = a < 1 ? 1 : (a > (kb0 + 3) / 4 ? (kb0 + 3) / 4 : a);
  int b = 0;
  if (kb1 > 0) {
    b = want - a;
    b = b < 1 ? 1 : (b > (kb1 + 3) / 4 ? (kb1 + 3) / 4 : b);
  }
  *s0 = a;
  *s1 = b;
}

}  // namespace dense

// shared with attn_mix.cu
int make_tmap_bf16_box64(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, int64_t pitch, uint32_t box_rows) {
  return dense::make_tmap_bf16_2d(map, ptr, cols, rows, pitch, box_rows);
}

}  // namespace fr

using namespace fr;

// Column ranges as the kernels get them; FR_ERR_BAD_ARG when they do not tile the columns as the header says.
static int check_segs(const fr_out_segment* segs, int n_segs, int N, dense::Segs* sg) {
  FR_CHECK_ARG(segs && n_segs > 0 && n_segs <= dense::kMaxSegs);
  sg->n = n_segs;
  for (int i = 0; i < n_segs; ++i) {
    const fr_out_segment& s = segs[i];
    const int end = i + 1 < n_segs ? segs[i + 1].n0 : N;
    FR_CHECK_ARG(s.out && s.n0 % 32 == 0 && s.n > 0 && s.kind >= 0 && s.kind <= FR_SEG_GELU_MUL);
    FR_CHECK_ARG(s.n0 < end && (i > 0 || s.n0 == 0));
    FR_CHECK_ARG(s.kind != FR_SEG_GELU_MUL || s.mul);
    if (dense::paired(s))
      FR_CHECK_ARG(s.n0 % 64 == 0 && (end - s.n0) % 64 == 0 && 2 * s.n <= end - s.n0);
    else
      FR_CHECK_ARG(s.n <= end - s.n0);
    sg->s[i] = s;
  }
  return FR_OK;
}

extern "C" int fr_dense_proj(int dtype, const void* a, int64_t lda, const void* w, int64_t ldw, int M, int N, int K,
                             const fr_out_segment* segs, int n_segs, int algo, cudaStream_t stream) {
  FR_CHECK_ARG((dtype == 0 || dtype == 1) && M >= 0 && N > 0);
  if (M == 0) return FR_OK;
  FR_CHECK_ARG(dense::operand_ok(a, lda, K) && dense::operand_ok(w, ldw, K) && N % 4 == 0);
  dense::Segs sg{};
  if (check_segs(segs, n_segs, N, &sg) != FR_OK) return FR_ERR_BAD_ARG;
  if (algo == 0) algo = M <= 8 ? 1 : 2;
  if (algo == 1) {
    FR_CHECK_SUPPORTED(M <= 8);
    return dtype == 0 ? dense::launch_rows_proj<__nv_bfloat16>(a, lda, w, ldw, M, N, K, sg, stream)
                      : dense::launch_rows_proj<float>(a, lda, w, ldw, M, N, K, sg, stream);
  }
  if (dtype == 1) {
    dim3 grid(ceil_div(N, 64), ceil_div(M, 64));
    dense::dense_simt_proj_kernel<<<grid, 256, 0, stream>>>(static_cast<const float*>(a), lda, static_cast<const float*>(w),
                                                            ldw, M, N, K, sg);
    return launch_status();
  }
  dense::TcArgs g{};
  g.M = M;
  g.N = N;
  g.n_parts = 1;
  g.kb[0] = ceil_div(K, dense::kBlockK);
  g.segs = sg;
  fr_gated_part part{a, w, nullptr, lda, ldw, 0, K, 0};
  switch (dense::pick_block_n(M, N)) {
    case 256: return dense::launch_tc<256, dense::kEpiSegs>(g, &part, stream);
    case 128: return dense::launch_tc<128, dense::kEpiSegs>(g, &part, stream);
    default: return dense::launch_tc<64, dense::kEpiSegs>(g, &part, stream);
  }
}

extern "C" int fr_dense_proj_split(int dtype, const void* a, int64_t lda, const void* w, int64_t ldw, int M, int N, int K,
                                   const fr_out_segment* segs, int n_segs, float* partials, int n_splits, cudaStream_t stream) {
  FR_CHECK_ARG(M > 0 && M <= 65535 && N > 0 && partials && n_splits > 0);
  dense::Segs sg{};
  if (check_segs(segs, n_segs, N, &sg) != FR_OK) return FR_ERR_BAD_ARG;
  const fr_gated_part part{a, w, nullptr, lda, ldw, 0, K, 0};
  const int r = fr_dense_gated_add(dtype, &part, 1, partials, N, M, N, partials, n_splits, nullptr, 0, 0, stream);  // x is left alone
  if (r != FR_OK) return r;
  auto kern = dtype == 0 ? dense::dense_finish_kernel<__nv_bfloat16> : dense::dense_finish_kernel<float>;
  return launch_kernel(kern, dim3(ceil_div(N, 256), M), 256, 0, stream, M <= kPdlRows, static_cast<const float*>(partials), n_splits, M, N, sg);
}

extern "C" int fr_dense_gated_add_splits(int dtype, int M, int N, int K0, int K1) {
  if (dtype != 0 || M <= 8 || N <= 0 || K0 <= 0) return 0;
  int a, b;
  dense::plan_splits(M, N, ceil_div(K0, dense::kBlockK), K1 > 0 ? ceil_div(K1, dense::kBlockK) : 0, &a, &b);
  return a + b;
}

extern "C" int fr_dense_gated_add(int dtype, const fr_gated_part* parts, int n_parts, float* x, int64_t ldx, int M, int N,
                                  float* partials, int n_splits, void* copy, int64_t ldc, int algo, cudaStream_t stream) {
  FR_CHECK_ARG((dtype == 0 || dtype == 1) && parts && (n_parts == 1 || n_parts == 2) && M >= 0 && N > 0);
  if (M == 0) return FR_OK;
  FR_CHECK_ARG(x && ldx >= N && (copy == nullptr || (ldc >= N && partials == nullptr)));
  dense::Parts pt{};
  pt.n = n_parts;
  for (int p = 0; p < n_parts; ++p) {
    FR_CHECK_ARG(dense::operand_ok(parts[p].a, parts[p].lda, parts[p].K) &&
                 dense::operand_ok(parts[p].w, parts[p].ldw, parts[p].K));
    pt.p[p] = parts[p];
  }
  if (partials == nullptr) n_splits = 0;
  if (algo == 0) algo = (M <= 8 && n_splits == 0) ? 1 : 2;
  if (algo == 1) {
    FR_CHECK_SUPPORTED(M <= 8 && n_splits == 0);
    return dtype == 0 ? dense::launch_rows_gated<__nv_bfloat16>(pt, x, ldx, M, N, copy, ldc, stream)
                      : dense::launch_rows_gated<float>(pt, x, ldx, M, N, copy, ldc, stream);
  }
  if (dtype == 1) {
    FR_CHECK_SUPPORTED(n_splits == 0);
    dim3 grid(ceil_div(N, 64), ceil_div(M, 64));
    dense::dense_simt_gated_kernel<<<grid, 256, 0, stream>>>(pt, x, ldx, M, N, static_cast<float*>(copy), ldc);
    return launch_status();
  }
  dense::TcArgs g{};
  g.M = M;
  g.N = N;
  g.n_parts = n_parts;
  g.x = x;
  g.ldx = ldx;
  g.copy = static_cast<__nv_bfloat16*>(copy);
  g.ldc = ldc;
  for (int p = 0; p < n_parts; ++p) {
    g.kb[p] = ceil_div(parts[p].K, dense::kBlockK);
    g.gate[p] = static_cast<const __nv_bfloat16*>(parts[p].gate);
    g.ldg[p] = parts[p].ldg;
  }
  if (n_splits > 0) {
    dense::plan_splits(M, N, g.kb[0], n_parts > 1 ? g.kb[1] : 0, &g.splits[0], &g.splits[1]);
    FR_CHECK_ARG(g.splits[0] > 0 && g.splits[0] + g.splits[1] == n_splits && (n_parts == 1 || g.splits[1] > 0));
    g.partials = partials;
    return dense::launch_tc<64, dense::kEpiPartial>(g, parts, stream);
  }
  switch (dense::pick_block_n(M, N)) {
    case 256: return dense::launch_tc<256, dense::kEpiAdd>(g, parts, stream);
    case 128: return dense::launch_tc<128, dense::kEpiAdd>(g, parts, stream);
    default: return dense::launch_tc<64, dense::kEpiAdd>(g, parts, stream);
  }
}
