// bf16 prompts of the matrix-state recurrences (fr_linear_scan in the header) on tcgen05, in chunks of 128 tokens.
// With r_i the sum of the log decays of the chunk's tokens after its first (r_0 = 0), u_j the value that enters the state
// (step_j v_j, or v_j) and a_0 the decay of the first token:
//
//     decay per head:     P_ij = e^(r_i - r_j) q_i . k_j   (j <= i)           O = e^r (Q (a_0 S)) + P U
//                         S <- e^(r_last) a_0 S + K^T (e^(r_last - r_j) u_j)
//     decay per channel:  q~_i = e^(r_i - m) q_i,  k~_j = e^(m - r_j) k_j,  P = mask(Q~ K~^T),  O = Q~ S' + P U
//                         S' = e^m a_0 S,  S <- e^(r_last - m) (S' + K~^T U),  m = r_last / 2
//
// The second form needs |r_last| below what e^(m - r) can hold. Heads of a request that leave this range anywhere are
// flagged and left to the token-by-token kernel.
//
// Decays, factors, masks and the state are fp32. What is not bf16 to begin with (q~, k~, scaled values, P, S') enters the
// tensor cores as a sum of two bf16 numbers, 16 significant bits, in two or three products.
//
//   head_factor_kernel     decay per head: e^r and its relatives, one warp per chunk and head
//   channel_factor_kernel  decay per channel: the low-rank decays, q~ and k~ of every chunk and head
//   chunk_kernel           one CTA: one head, up to 64 columns of V and S, one segment of a request, chunk after chunk. S
//                          lives in registers (thread = row of S and a quarter of the columns). Warps 0..15 work on
//                          operands, mask, state and output, warp 16 issues tcgen05.mma, warp 17 TMA. Scores, tiles and
//                          operands are one chunk ahead of the output.
//
// Long prompts are cut into segments that run side by side: a first launch finds the state that each segment adds and its
// total decay, the second starts every segment from the combination of those before it.
#include "fr_common.cuh"
#include "linear_scan.cuh"
#include "sm100_ptx.cuh"

namespace fr {

int* device_status_ptr();  // capi.cu
int make_tmap_bf16_box64(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, int64_t pitch,
                         uint32_t box_rows);  // dense_proj.cu

namespace scan {

constexpr int kChunk = 128;            // tokens (UMMA M)
constexpr int kVb = 64;                // columns of V per CTA: one swizzle span
constexpr int kBox = kChunk * 128;     // bytes of a [128 x 64] bf16 tile
constexpr int kCompute = 512;          // threads of the compute warps
constexpr int kThreads = kCompute + 64;
constexpr float kLog2e = 1.4426950408889634f;
// largest -r_last (in powers of two) per channel: e^(+-r_last / 2), the products of visible pairs and the state's sums stay
// far inside 2^+-126 (scores of later keys may not: they are replaced, not multiplied, by zero)
constexpr float kMaxChannel = 160.f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two values as packed bf16, and what is left of them
__device__ __forceinline__ uint32_t split2(float a, float b, uint32_t& lo) {
  const uint32_t hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16lo(hi), b - bf16hi(hi));
  return hi;
}
__device__ __forceinline__ uint32_t split2(uint64_t v, uint32_t& lo) {
  float a, b;
  unpack2(v, a, b);
  const uint32_t hi = pack_bf16(a, b);
  unpack2(fma2(pack2(bf16lo(hi), bf16hi(hi)), dup2(-1.0f), v), a, b);
  lo = pack_bf16(a, b);
  return hi;
}

// log2(1 + e^z): the logarithm's series where 1 + e^-|z| would lose the small term
__device__ __forceinline__ float softplus_log2(float z) {
  const float e = ex2(-fabsf(z) * kLog2e);
  const float series = kLog2e * e * (1.0f - e * (0.5f - e * (1.0f / 3.0f - 0.25f * e)));
  return fmaf(fmaxf(z, 0.f), kLog2e, e < 0.0156f ? series : __log2f(1.0f + e));
}

// Factors of one chunk and head.
struct HeadFactors {
  float r[kChunk];    // r_i (log2)
  float l[kChunk];    // r_i counted from the block of 32 tokens that i is in
  float c[kChunk];    // log2(step_j) - l_j
  float x[kChunk];    // step_j e^(r_last - r_j)
  float y[kChunk];    // step_j e^(r_e - r_j), e the last of j's block of 32 tokens
  float first, end;   // a_0, e^(r_last)
  float pad_[2];
};
struct ChannelFactors {  // per row of S
  float first[kChunk];   // e^m a_0
  float end[kChunk];     // e^(r_last - m)
};

struct ChunkPlan {
  int boxes;     // 64-column boxes of a q / k row
  int seg_len;   // tokens per segment (a multiple of kChunk)
  int segs;      // segments of the longest request
  int v_blocks;
  int smem;
};

struct ChunkArgs {
  fr_linear_scan a;
  ChunkPlan pl;
  int min_tokens;      // shorter requests are left alone
  void* factors;       // [chunk, head]
  __nv_bfloat16* qk;   // CHANNEL: q~ hi, q~ lo, k~ hi, k~ lo, each [T, heads * dim]
  int64_t qk_stride;   // elements of one of them
  int32_t* flags;      // CHANNEL: [request, head] left to the token-by-token kernel
  float* seg_state;    // [request, segment, head][dim][state cols]
  float* seg_decay;    // [request, segment, head][dim]
  float* start_state;  // [request, head][dim][state cols]
};

// Number of a request's first chunk: requests take ceil(tokens / 128) numbers each without overlapping.
__device__ __forceinline__ int64_t first_chunk(int q0, int b) { return q0 / kChunk + b; }

// ---------------------------------------------------------------------------
constexpr int kFactorHeads = 8;
__global__ void __launch_bounds__(kFactorHeads * 32)
head_factor_kernel(const __grid_constant__ ChunkArgs g) {
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const fr_linear_scan& a = g.a;
  const int b = blockIdx.z, h = blockIdx.y * kFactorHeads + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int q0 = a.qo_indptr[b], q1 = a.qo_indptr[b + 1];
  const int t = q0 + blockIdx.x * kChunk, n = min(kChunk, q1 - t);
  if (h >= a.heads || t >= q1) return;
  HeadFactors* f = static_cast<HeadFactors*>(g.factors) + (first_chunk(q0, b) + blockIdx.x) * a.heads + h;
  const float rate = -a.rate[h] * kLog2e;
  float step[4], la[4], sum = 0.f, first = 0.f;  // four tokens per lane
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int i = lane * 4 + e;
    step[e] = i < n ? head_step(a, t + i, h) : 0.f;
    la[e] = rate * step[e];
  }
  if (lane == 0) {
    first = ex2(la[0]);
    la[0] = 0.f;
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) sum += la[e];
  float x = sum;
#pragma unroll
  for (int o = 1; o < 32; o *= 2) {
    const float y = __shfl_up_sync(0xffffffffu, x, o);
    if (lane >= o) x += y;
  }
  const float last = __shfl_sync(0xffffffffu, x, 31);
  float z = sum;  // the same within a block: differences of nearby tokens keep their digits however strong the decay
#pragma unroll
  for (int o = 1; o < 8; o *= 2) {
    const float y = __shfl_up_sync(0xffffffffu, z, o);
    if ((lane & 7) >= o) z += y;
  }
  const float block_end = __shfl_sync(0xffffffffu, z, lane | 7);
  float r = x - sum, l = z - sum, fr[4], fl[4], fc[4], fx[4], fy[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    r += la[e];
    l += la[e];
    fr[e] = r;
    fl[e] = l;
    fc[e] = log2f(step[e]) - l;  // -inf past the end: no weight
    fx[e] = step[e] * ex2(last - r);
    fy[e] = step[e] * ex2(block_end - l);
  }
  *reinterpret_cast<float4*>(f->r + lane * 4) = make_float4(fr[0], fr[1], fr[2], fr[3]);
  *reinterpret_cast<float4*>(f->l + lane * 4) = make_float4(fl[0], fl[1], fl[2], fl[3]);
  *reinterpret_cast<float4*>(f->c + lane * 4) = make_float4(fc[0], fc[1], fc[2], fc[3]);
  *reinterpret_cast<float4*>(f->x + lane * 4) = make_float4(fx[0], fx[1], fx[2], fx[3]);
  *reinterpret_cast<float4*>(f->y + lane * 4) = make_float4(fy[0], fy[1], fy[2], fy[3]);
  if (lane == 0) *reinterpret_cast<float4*>(&f->first) = make_float4(first, ex2(last), 0.f, 0.f);
}

// One chunk of one head: a thread has two channels and a share of the tokens.
constexpr int kPrepThreads = 256;
__global__ void __launch_bounds__(kPrepThreads)
channel_factor_kernel(const __grid_constant__ ChunkArgs g) {
  extern __shared__ __align__(16) float sm[];
  const fr_linear_scan& a = g.a;
  const int pairs = a.dim / 2;
  int parts = 1;
  while (parts * 2 * pairs <= kPrepThreads && parts < 32) parts *= 2;
  const int tp = kChunk / parts;
  float* s_la = sm;                         // [128][dim]
  float* s_low = s_la + kChunk * a.dim;     // [rank][128]
  float* s_part = s_low + kChunk * a.rank;  // [parts][dim]
  float* s_up = s_part + 2 * kPrepThreads;  // [rank][dim]
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y, tid = threadIdx.x;
  const int q0 = a.qo_indptr[b], q1 = a.qo_indptr[b + 1];
  const int t = q0 + blockIdx.x * kChunk;
  if (t >= q1) return;
  const int n = min(kChunk, q1 - t);
  for (int e = tid; e < kChunk * a.rank; e += kPrepThreads) {
    const int i = e / a.rank, c = e % a.rank;
    s_low[c * kChunk + i] = i < n ? a.step[static_cast<int64_t>(t + i) * a.ldstep + c] : 0.f;
  }
  for (int e = tid; e < a.dim * a.rank; e += kPrepThreads)
    s_up[e % a.rank * a.dim + e / a.rank] = a.up[static_cast<int64_t>(h) * a.dim * a.rank + e];
  __syncthreads();
  const int part = tid / pairs, ch = 2 * (tid % pairs), i0 = part * tp, i1 = min(n, i0 + tp);
  const bool live = part < parts;
  if (live) {
    const int hc = h * a.dim + ch;
    const float b0 = a.step_bias[hc], b1 = a.step_bias[hc + 1], f = -a.inv_tau;
    float2 sum = make_float2(0.f, 0.f);
    for (int i = i0; i < i1; i += 4) {
      float z0[4], z1[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        z0[e] = b0;
        z1[e] = b1;
      }
      for (int r = 0; r < a.rank; ++r) {
        const float2 u = *reinterpret_cast<const float2*>(s_up + r * a.dim + ch);
        const float4 l4 = *reinterpret_cast<const float4*>(s_low + r * kChunk + i);
        const float low[4] = {l4.x, l4.y, l4.z, l4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          z0[e] = fmaf(u.x, low[e], z0[e]);
          z1[e] = fmaf(u.y, low[e], z1[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (i + e >= i1) break;
        const float2 la = make_float2(softplus_log2(-z0[e]) * f, softplus_log2(-z1[e]) * f);
        *reinterpret_cast<float2*>(s_la + (i + e) * a.dim + ch) = la;
        if (i + e > 0) {
          sum.x += la.x;
          sum.y += la.y;
        }
      }
    }
    *reinterpret_cast<float2*>(s_part + part * a.dim + ch) = sum;
  }
  __syncthreads();
  if (!live) return;
  float2 r = make_float2(0.f, 0.f), last = r;
  for (int p = 0; p < parts; ++p) {
    const float2 d = *reinterpret_cast<const float2*>(s_part + p * a.dim + ch);
    if (p < part) {
      r.x += d.x;
      r.y += d.y;
    }
    last.x += d.x;
    last.y += d.y;
  }
  // out of range: flagged; what is written stays finite (a neighbour's tile may hold these rows, times zero)
  const bool wide = fminf(last.x, last.y) < -kMaxChannel;
  const float m0 = 0.5f * fmaxf(last.x, -kMaxChannel), m1 = 0.5f * fmaxf(last.y, -kMaxChannel);
  if (part == 0) {
    const float2 la = *reinterpret_cast<const float2*>(s_la + ch);
    ChannelFactors* f = static_cast<ChannelFactors*>(g.factors) + (first_chunk(q0, b) + blockIdx.x) * a.heads + h;
    *reinterpret_cast<float2*>(f->first + ch) = make_float2(ex2(la.x + m0), ex2(la.y + m1));
    *reinterpret_cast<float2*>(f->end + ch) = make_float2(ex2(last.x - m0), ex2(last.y - m1));
    if (wide) g.flags[b * a.heads + h] = 1;
  }
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + static_cast<int64_t>(t) * a.ldq + h * a.dim + ch;
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + static_cast<int64_t>(t) * a.ldk + h * a.dim + ch;
  const int64_t ld = static_cast<int64_t>(a.heads) * a.dim;
  __nv_bfloat16* out = g.qk + t * ld + h * a.dim + ch;
#pragma unroll 8
  for (int i = i0; i < i1; ++i) {
    if (i > 0) {
      const float2 d = *reinterpret_cast<const float2*>(s_la + i * a.dim + ch);
      r.x += d.x;
      r.y += d.y;
    }
    const uint32_t qv = *reinterpret_cast<const uint32_t*>(qp + i * a.ldq), kv = *reinterpret_cast<const uint32_t*>(kp + i * a.ldk);
    const float e0 = fminf(fmaxf(r.x - m0, -kMaxChannel / 2), kMaxChannel / 2), e1 = fminf(fmaxf(r.y - m1, -kMaxChannel / 2), kMaxChannel / 2);
    uint32_t lo;
    __nv_bfloat16* o = out + i * ld;
    *reinterpret_cast<uint32_t*>(o) = split2(bf16lo(qv) * a.scale * ex2(e0), bf16hi(qv) * a.scale * ex2(e1), lo);
    *reinterpret_cast<uint32_t*>(o + g.qk_stride) = lo;
    *reinterpret_cast<uint32_t*>(o + 2 * g.qk_stride) = split2(bf16lo(kv) * ex2(-e0), bf16hi(kv) * ex2(-e1), lo);
    *reinterpret_cast<uint32_t*>(o + 3 * g.qk_stride) = lo;
  }
}

// ---------------------------------------------------------------------------
// Shared memory: tiles of q and k (CHANNEL: hi and lo each), kSets of v, S' hi and lo, HEAD: scaled v hi and lo; factors.
constexpr int kSets = 3;
__host__ __device__ __forceinline__ int tile_smem(bool channel, int boxes, int dim) {
  return (channel ? 4 : 2) * boxes * kBox + kSets * kBox + (channel ? 0 : 2 * kBox) + 2 * dim * 128;
}
template <bool CHANNEL>
struct FactorsOf {
  using type = HeadFactors;
};
template <>
struct FactorsOf<true> {
  using type = ChannelFactors;
};
constexpr int kTailSmem = kSets * static_cast<int>(sizeof(HeadFactors)) + 128;
static_assert(sizeof(HeadFactors) % 16 == 0 && sizeof(ChannelFactors) % 16 == 0 && sizeof(ChannelFactors) <= sizeof(HeadFactors));

// f(0), .. f(n - 1), unrolled for the usual numbers of steps (the products are short: issuing them would pace the tensor
// cores)
template <class F>
__device__ __forceinline__ void steps(int n, F&& f) {
  if (n == 8) {
#pragma unroll
    for (int k = 0; k < 8; ++k) f(k);
  } else if (n == 4) {
#pragma unroll
    for (int k = 0; k < 4; ++k) f(k);
  } else {
#pragma unroll 1
    for (int k = 0; k < n; ++k) f(k);
  }
}
// MN-major operand of 64-value blocks that are `lead` bytes apart
__device__ __forceinline__ uint64_t desc_mn(uint32_t addr, uint32_t lead) {
  return (ptx::smem_desc_sw128(addr) & ~(static_cast<uint64_t>(0x3fffu) << 16)) | static_cast<uint64_t>((lead >> 4) & 0x3fffu) << 16;
}

struct ChunkMaps {
  CUtensorMap v, q, k, q_lo, k_lo, out;
};

template <bool CHANNEL, bool STATE_ONLY>
__global__ void __launch_bounds__(kThreads, 1)
chunk_kernel(const __grid_constant__ ChunkMaps maps, const __grid_constant__ ChunkArgs g, int* status) {
  using Factors = typename FactorsOf<CHANNEL>::type;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const fr_linear_scan& a = g.a;
  const ChunkPlan& pl = g.pl;
  const int kq = pl.boxes * kBox;
  const uint32_t off_q = 0, off_k = (CHANNEL ? 2u : 1u) * kq;  // CHANNEL: hi, lo
  const uint32_t off_v = 2u * off_k;                           // kSets tiles; a full chunk's output takes its v's place
  const uint32_t off_x = off_v + kSets * kBox;                 // HEAD: scaled v hi, lo
  const uint32_t off_s = CHANNEL ? off_x : off_x + 2u * kBox;
  const uint32_t s_bytes = a.dim * 128;
  Factors* fac = reinterpret_cast<Factors*>(smem + off_s + 2 * s_bytes);
  uint64_t* bars = reinterpret_cast<uint64_t*>(fac + kSets);
  const uint32_t bar_v = ptx::smem_u32(bars);          // [kSets]
  const uint32_t bar_qk = bar_v + 8 * kSets, bar_g = bar_qk + 8, bar_su = bar_qk + 16, bar_o = bar_qk + 24;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + kSets + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool compute = tid < kCompute, issuer = tid == kCompute, loader = tid == kCompute + 32;
  ptx::griddep_wait();
  const int h = blockIdx.x / pl.v_blocks, c0 = (blockIdx.x % pl.v_blocks) * kVb;
  const int b = blockIdx.z, seg = blockIdx.y;
  const int q0 = a.qo_indptr[b], q1 = a.qo_indptr[b + 1];
  const int t_begin = q0 + seg * pl.seg_len;
  if (q1 - q0 < g.min_tokens || t_begin >= q1) return;
  if (STATE_ONLY && t_begin + pl.seg_len >= q1) return;  // nothing follows the last segment
  if (CHANNEL && g.flags[b * a.heads + h] != 0) return;
  const int t_end = min(t_begin + pl.seg_len, q1);
  const int kh = h / (a.heads / a.key_heads);
  const int vb = min(kVb, a.vdim - c0);
  const int vp = state_cols(a.vdim);

  if (tid == 0) {
    for (int i = 0; i < kSets + 4; ++i) ptx::mbar_init(bar_v + 8 * i, 1);
    *abort_flag = 0;
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&maps.v);
    ptx::prefetch_tmap(&maps.q);
    ptx::prefetch_tmap(&maps.k);
  }
  if (warp == kCompute / 32) {
    __syncwarp();
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), 512);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  ptx::griddep_launch_dependents();  // not before the tensor memory is taken
  const uint32_t tmem = *tmem_slot;
  // scores and P; Q S' with S' hi and lo side by side; K^T U (HEAD: with U hi and lo); P U (CHANNEL: added to Q S' hi)
  const uint32_t col_p = tmem, col_in = tmem + 128, col_su = tmem + 256, col_pu = CHANNEL ? col_in : tmem + 384;
  const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;
  const Factors* factors = static_cast<const Factors*>(g.factors) + (first_chunk(q0, b) + seg * (pl.seg_len / kChunk)) * a.heads + h;

  // ---- TMA and tcgen05.mma, one thread each --------------------------------------------------------------
  auto load_v = [&](int it) {
    const int set = it % kSets;
    ptx::mbar_expect_tx(bar_v + 8 * set, kBox + sizeof(Factors));
    ptx::tma_load_2d(base + off_v + set * kBox, &maps.v, h * a.vdim + c0, t_begin + it * kChunk, bar_v + 8 * set);
    ptx::bulk_load(ptx::smem_u32(fac + set), factors + static_cast<int64_t>(it) * a.heads, sizeof(Factors), bar_v + 8 * set);
  };
  auto load_qk = [&](int it) {
    const int t = t_begin + it * kChunk;
    ptx::mbar_expect_tx(bar_qk, (STATE_ONLY ? 1 : 2) * off_k);
    for (int x = 0; x < pl.boxes; ++x) {
      const int col = kh * a.dim + x * 64;
      if (!STATE_ONLY) ptx::tma_load_2d(base + off_q + x * kBox, &maps.q, col, t, bar_qk);
      ptx::tma_load_2d(base + off_k + x * kBox, &maps.k, col, t, bar_qk);
      if (CHANNEL) {
        if (!STATE_ONLY) ptx::tma_load_2d(base + off_q + kq + x * kBox, &maps.q_lo, col, t, bar_qk);
        ptx::tma_load_2d(base + off_k + kq + x * kBox, &maps.k_lo, col, t, bar_qk);
      }
    }
  };
  auto issue_scores = [&] {
    constexpr uint32_t idesc = ptx::make_idesc(1u, 1u, kChunk, kChunk);
    const uint64_t qd = ptx::smem_desc_sw128(base + off_q), kd = ptx::smem_desc_sw128(base + off_k);
    const uint64_t lo = kq >> 4;
    steps(a.dim / 16, [&](int k) {
      const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3);
      ptx::mma_f16(col_p, qd + o, kd + o, idesc, k > 0 ? 1u : 0u);
      if (CHANNEL) {
        ptx::mma_f16(col_p, qd + o, kd + lo + o, idesc, 1u);
        ptx::mma_f16(col_p, qd + lo + o, kd + o, idesc, 1u);
      }
    });
    ptx::tc_commit(bar_g);
  };
  auto wait_bar = [&](uint32_t bar, uint32_t parity, int site) {  // whole warps
    if (lane == 0) ptx::mbar_wait(bar, parity, abort_flag, status, site);
    __syncwarp();
    ptx::tc_fence_after();
  };

  // ---- S: row of the state and a quarter of the columns --------------------------------------------------
  const int row = tid & 127, quarter = (tid >> 7) & 3, col0 = quarter * 16;
  const bool state_thread = compute && row < a.dim;
  const bool my_cols = col0 < vb;  // vb is a multiple of 16
  float s[16];
  float decay_all = 1.0f;
  const int64_t per = static_cast<int64_t>(a.dim) * vp;
  const int64_t here = static_cast<int64_t>(row) * vp + c0 + col0;
  {
    const int64_t seg0 = static_cast<int64_t>(b) * pl.segs;
#pragma unroll
    for (int c = 0; c < 16; ++c) s[c] = 0.f;
    if (state_thread && my_cols) {
      if (seg == 0) {
        const bool fresh = a.pos[q0] == 0;
        const bool saved = !STATE_ONLY && pl.segs > 1 && q1 - q0 > pl.seg_len;
        float* keep = g.start_state + (static_cast<int64_t>(b) * a.heads + h) * per + here;
        const float* src = saved ? keep : a.state + (a.state_slots[b] * a.heads + h) * per + here;
#pragma unroll
        for (int c = 0; c < 16; c += 4) {
          float4 v = make_float4(0, 0, 0, 0);
          if (saved || !fresh) v = *reinterpret_cast<const float4*>(src + c);
          s[c] = v.x; s[c + 1] = v.y; s[c + 2] = v.z; s[c + 3] = v.w;
          if (STATE_ONLY) *reinterpret_cast<float4*>(keep + c) = v;
        }
      } else if (!STATE_ONLY) {
        for (int r = 0; r < seg; ++r) {
          const int64_t id = (seg0 + r) * a.heads + h;
          const float d = r == 0 ? 0.f : g.seg_decay[id * a.dim + row];
#pragma unroll
          for (int c = 0; c < 16; c += 4) {
            const float4 v = *reinterpret_cast<const float4*>(g.seg_state + id * per + here + c);
            s[c] = fmaf(d, s[c], v.x); s[c + 1] = fmaf(d, s[c + 1], v.y);
            s[c + 2] = fmaf(d, s[c + 2], v.z); s[c + 3] = fmaf(d, s[c + 3], v.w);
          }
        }
      }
    }
  }
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;

  // Operands of a chunk: S' over the old state and its halves, scaled values; `x` keeps the raw values.
  auto operands = [&](int it, uint32_t (&x)[8]) {
    const int n = min(kChunk, t_end - (t_begin + it * kChunk)), set = it % kSets;
    wait_bar(bar_v + 8 * set, (it / kSets) & 1, 92);
    const Factors* f = fac + set;
    if (state_thread) {
      float first;
      if constexpr (CHANNEL) first = f->first[row];
      else first = f->first;
      decay_all *= first;
      uint8_t* dst = smem + off_s + row * 128;
#pragma unroll
      for (int c = 0; c < 16; ++c) s[c] *= first;
      if (!STATE_ONLY) {
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) hi[e] = split2(s[8 * y + 2 * e], s[8 * y + 2 * e + 1], lo[e]);
          const int o = ((quarter * 2 + y) ^ (row & 7)) << 4;
          *reinterpret_cast<uint4*>(dst + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(dst + s_bytes + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
    }
    uint8_t* vrow = smem + off_v + set * kBox + row * 128;
    const bool in = row < n;
    if (!in) {  // another request's values, or none
#pragma unroll
      for (int y = 0; y < 2; ++y) *reinterpret_cast<uint4*>(vrow + (((quarter * 2 + y) ^ (row & 7)) << 4)) = make_uint4(0, 0, 0, 0);
    }
    if constexpr (!CHANNEL) {
      const float w = f->x[row];
      uint8_t* dst = smem + off_x + row * 128;
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int o = ((quarter * 2 + y) ^ (row & 7)) << 4;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (in) v = *reinterpret_cast<const uint4*>(vrow + o);
        x[4 * y] = v.x; x[4 * y + 1] = v.y; x[4 * y + 2] = v.z; x[4 * y + 3] = v.w;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) hi[e] = split2(bf16lo(x[4 * y + e]) * w, bf16hi(x[4 * y + e]) * w, lo[e]);
        *reinterpret_cast<uint4*>(dst + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(dst + kBox + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
    ptx::fence_proxy_async_smem();
  };

  const int n_chunks = (t_end - t_begin + kChunk - 1) / kChunk;
  // A full chunk's output tile leaves by TMA (a partial one must not touch the rows or columns beside it).
  auto full_tile = [&](int it) { return !STATE_ONLY && vb == kVb && t_end - (t_begin + it * kChunk) >= kChunk; };
  auto store_tile = [&](int it) {
    ptx::tma_store_2d(&maps.out, base + off_v + (it % kSets) * kBox, h * a.vdim + c0, t_begin + it * kChunk);
    ptx::bulk_commit();
  };
  uint32_t x_now[8], x_next[8];
  if (loader) {
    load_v(0);
    load_qk(0);
    if (n_chunks > 1) load_v(1);
  }
  __syncwarp();
  if (issuer && !STATE_ONLY && ptx::mbar_wait(bar_qk, 0, abort_flag, status, 91)) issue_scores();
  __syncwarp();
  if (compute) operands(0, x_now);
  for (int it = 0; it < n_chunks; ++it) {
    const int t = t_begin + it * kChunk, n = min(kChunk, t_end - t);
    const int set = it % kSets, ph = it & 1;
    const Factors* f = fac + set;
    const int k_tok = (n + 15) / 16;  // steps of 16 tokens
    const bool more = it + 1 < n_chunks;
    ptx::tc_fence_before();
    __syncthreads();
    if (*abort_flag) break;
    if (warp == kCompute / 32 + 1) {
      if (loader) {
        if (it > 0 && full_tile(it - 1)) store_tile(it - 1);
        if (more && ptx::mbar_wait(bar_su, ph, abort_flag, status, 97)) {  // q's and k's tiles are free
          load_qk(it + 1);
          if (it + 2 < n_chunks) {  // and the v tile of the chunk before, once its output has left
            ptx::bulk_wait_read<0>();
            load_v(it + 2);
          }
        }
      }
      __syncwarp();
      continue;
    }
    if (issuer) {
      ptx::tc_fence_after();
      constexpr uint32_t kMnB = 1u << 16, kMnA = 1u << 15;  // operands that lie MN-major
      constexpr uint32_t idesc_pair = ptx::make_idesc(1u, 1u, kChunk, 2 * kVb) | kMnB;
      constexpr uint32_t idesc_one = ptx::make_idesc(1u, 1u, kChunk, kVb) | kMnB;
      if (!STATE_ONLY) {
        const uint64_t qd = ptx::smem_desc_sw128(base + off_q), qlo = qd + (kq >> 4), sd = desc_mn(base + off_s, s_bytes);
        steps(a.dim / 16, [&](int k) {
          const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3), so = k * 128u;
          ptx::mma_f16(col_in, qd + o, sd + so, idesc_pair, k > 0 ? 1u : 0u);
          if (CHANNEL) ptx::mma_f16(col_in, qlo + o, sd + so, idesc_pair, 1u);
        });
      } else {
        ptx::mbar_wait(bar_qk, ph, abort_flag, status, 96);
      }
      // A = K^T: rows of S by tokens, a second box of rows for more than 64 (else the first once more, unused)
      const uint64_t kt = desc_mn(base + off_k, pl.boxes > 1 ? kBox : 0);
      const uint64_t ud = desc_mn(base + (CHANNEL ? off_v + set * kBox : off_x), kBox);
      steps(k_tok, [&](int k) {
        const uint64_t o = k * 128u;
        ptx::mma_f16(col_su, kt + o, ud + o, (CHANNEL ? idesc_one : idesc_pair) | kMnA, k > 0 ? 1u : 0u);
        if (CHANNEL) ptx::mma_f16(col_su, kt + (kq >> 4) + o, ud + o, idesc_one | kMnA, 1u);
      });
      ptx::tc_commit(bar_su);
    }
    __syncwarp();

    // ---- P as two bf16 halves over the scores, 32 columns per thread: [16 hi | 16 lo] ------------------
    if (!STATE_ONLY) {
      if (compute) {
        wait_bar(bar_g, ph, 93);
        if (quarter * 32 < n) {
          uint32_t p[32];
          if (quarter > (warp & 3)) {  // keys after every query of this warp
#pragma unroll
            for (int c = 0; c < 32; ++c) p[c] = 0u;
          } else if (quarter < (warp & 3)) {  // before every query: e^(r_i - r_j) in two factors, both at most one
            uint32_t gv[32];
            ptx::tmem_ld_32x32(col_p + lane_off + quarter * 32, gv);
            uint64_t ai = 0;
            if constexpr (!CHANNEL) ai = dup2(ex2(f->r[row] - f->r[quarter * 32 + 31]));
            ptx::tmem_ld_wait();
#pragma unroll
            for (int c4 = 0; c4 < 8; ++c4) {
              uint64_t v0 = pack2(__uint_as_float(gv[4 * c4]), __uint_as_float(gv[4 * c4 + 1]));
              uint64_t v1 = pack2(__uint_as_float(gv[4 * c4 + 2]), __uint_as_float(gv[4 * c4 + 3]));
              if constexpr (!CHANNEL) {
                const ulonglong2 yj = *reinterpret_cast<const ulonglong2*>(f->y + quarter * 32 + 4 * c4);
                v0 = mul2(mul2(v0, yj.x), ai);
                v1 = mul2(mul2(v1, yj.y), ai);
              }
              p[2 * c4] = split2(v0, p[16 + 2 * c4]);
              p[2 * c4 + 1] = split2(v1, p[16 + 2 * c4 + 1]);
            }
          } else {
            uint32_t gv[32];
            ptx::tmem_ld_32x32(col_p + lane_off + quarter * 32, gv);
            float ri = 0.f;
            if constexpr (!CHANNEL) ri = f->l[row];
            ptx::tmem_ld_wait();
#pragma unroll
            for (int c4 = 0; c4 < 8; ++c4) {
              float v[4] = {__uint_as_float(gv[4 * c4]), __uint_as_float(gv[4 * c4 + 1]), __uint_as_float(gv[4 * c4 + 2]),
                            __uint_as_float(gv[4 * c4 + 3])};
              const int j = quarter * 32 + 4 * c4;
              if constexpr (!CHANNEL) {
                const float4 cj = *reinterpret_cast<const float4*>(f->c + j);
                v[0] *= ex2(ri + cj.x); v[1] *= ex2(ri + cj.y); v[2] *= ex2(ri + cj.z); v[3] *= ex2(ri + cj.w);
              }
#pragma unroll
              for (int e = 0; e < 4; ++e) v[e] = j + e <= row ? v[e] : 0.f;
              p[2 * c4] = split2(v[0], v[1], p[16 + 2 * c4]);
              p[2 * c4 + 1] = split2(v[2], v[3], p[16 + 2 * c4 + 1]);
            }
          }
          ptx::tmem_st_32x32(col_p + lane_off + quarter * 32, p);
          ptx::tmem_st_wait();
        }
        ptx::tc_fence_before();
      }
      asm volatile("bar.sync 1, %0;" ::"n"(kCompute + 32) : "memory");  // all but the loader's warp
      if (issuer) {
        ptx::tc_fence_after();
        constexpr uint32_t idesc_one = ptx::make_idesc(1u, 1u, kChunk, kVb) | (1u << 16);
        const uint64_t vd = desc_mn(base + off_v + set * kBox, kBox);
        if (CHANNEL) ptx::mbar_wait(bar_su, ph, abort_flag, status, 100);  // Q S' is in place: products of another shape follow
        steps(k_tok, [&](int k) {
          const uint32_t pc = col_p + (k >> 1) * 32 + (k & 1) * 8;
          ptx::mma_f16_ts(col_pu, pc, vd + k * 128u, idesc_one, CHANNEL || k > 0 ? 1u : 0u);
          ptx::mma_f16_ts(col_pu, pc + 16, vd + k * 128u, idesc_one, 1u);
        });
        ptx::tc_commit(bar_o);
        if (more && ptx::mbar_wait(bar_o, ph, abort_flag, status, 99) &&  // the next scores overwrite P
            ptx::mbar_wait(bar_qk, ph ^ 1, abort_flag, status, 98))
          issue_scores();
      }
      __syncwarp();
    }

    // ---- new state, operands of the next chunk, output ------------------------------------------------
    if (compute) {
      wait_bar(bar_su, ph, 94);
      uint32_t v[16], y[16];
      ptx::tmem_ld_32x16(col_su + lane_off + col0, v);
      if (!CHANNEL) ptx::tmem_ld_32x16(col_su + kVb + lane_off + col0, y);
      ptx::tmem_ld_wait();
      if (state_thread) {
        float end;
        if constexpr (CHANNEL) end = f->end[row];
        else end = f->end;
#pragma unroll
        for (int c = 0; c < 16; ++c)
          s[c] = CHANNEL ? end * (s[c] + __uint_as_float(v[c])) : fmaf(end, s[c], __uint_as_float(v[c]) + __uint_as_float(y[c]));
        decay_all *= end;
      }
      __syncwarp();
      if (more) operands(it + 1, x_next);
      if (!STATE_ONLY) {
        ptx::tmem_ld_32x16(col_in + kVb + lane_off + col0, y);  // Q S', with the low halves
        if (!CHANNEL) {
          ptx::tmem_ld_32x16(col_in + lane_off + col0, v);
          ptx::tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) y[e] = __float_as_uint(__uint_as_float(y[e]) + __uint_as_float(v[e]));
        }
        wait_bar(bar_o, ph, 95);
        ptx::tmem_ld_32x16(col_pu + lane_off + col0, v);
        ptx::tmem_ld_wait();
        if (row < n && my_cols) {
          const bool tile = full_tile(it);
          uint8_t* stage = smem + off_v + set * kBox + row * 128;
          __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + static_cast<int64_t>(t + row) * a.ldo + h * a.vdim + c0 + col0;
          float er = 0.f;
          if constexpr (!CHANNEL) er = ex2(f->r[row]);
          uint32_t w[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            float y0 = __uint_as_float(v[2 * e]), y1 = __uint_as_float(v[2 * e + 1]);
            if (CHANNEL) {
              y0 += __uint_as_float(y[2 * e]);
              y1 += __uint_as_float(y[2 * e + 1]);
            } else {
              y0 = fmaf(skip, bf16lo(x_now[e]), a.scale * fmaf(er, __uint_as_float(y[2 * e]), y0));
              y1 = fmaf(skip, bf16hi(x_now[e]), a.scale * fmaf(er, __uint_as_float(y[2 * e + 1]), y1));
            }
            w[e] = pack_bf16(y0, y1);
          }
          *reinterpret_cast<uint4*>(tile ? stage + (((quarter * 2) ^ (row & 7)) << 4) : reinterpret_cast<uint8_t*>(out)) =
              make_uint4(w[0], w[1], w[2], w[3]);
          *reinterpret_cast<uint4*>(tile ? stage + (((quarter * 2 + 1) ^ (row & 7)) << 4) : reinterpret_cast<uint8_t*>(out + 8)) =
              make_uint4(w[4], w[5], w[6], w[7]);
          ptx::fence_proxy_async_smem();
        }
        __syncwarp();
#pragma unroll
        for (int e = 0; e < 8; ++e) x_now[e] = x_next[e];
      }
    }
  }

  if (state_thread && my_cols) {
    float* dst = nullptr;
    if (STATE_ONLY) {
      const int64_t id = (static_cast<int64_t>(b) * pl.segs + seg) * a.heads + h;
      dst = g.seg_state + id * per;
      if (quarter == 0 && c0 == 0) g.seg_decay[id * a.dim + row] = decay_all;
    } else if (t_end == q1) {
      dst = a.state + (a.state_slots[b] * a.heads + h) * per;
    }
    if (dst != nullptr) {
#pragma unroll
      for (int c = 0; c < 16; c += 4) *reinterpret_cast<float4*>(dst + here + c) = make_float4(s[c], s[c + 1], s[c + 2], s[c + 3]);
    }
  }
  ptx::tc_fence_before();
  __syncthreads();
  if (loader) {
    if (!*abort_flag && full_tile(n_chunks - 1)) store_tile(n_chunks - 1);
    ptx::bulk_wait_all();
  }
  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == kCompute / 32) {
    ptx::tc_fence_after();
    ptx::tmem_dealloc(tmem, 512);
  }
}

// ---------------------------------------------------------------------------
static int channel_smem(const fr_linear_scan& a) { return (kChunk * (a.dim + a.rank) + 2 * kPrepThreads + a.rank * a.dim) * 4; }

static bool plan_chunks(const fr_linear_scan& a, int n_req, int longest, ChunkPlan* pl) {
  if (a.dim % 16 != 0 || a.vdim % 16 != 0 || a.dim > kChunk) return false;
  if (a.decay == FR_DECAY_CHANNEL && channel_smem(a) > 200 * 1024) return false;
  const bool channel = a.decay == FR_DECAY_CHANNEL;
  pl->boxes = (a.dim + 63) / 64;
  pl->v_blocks = ceil_div(a.vdim, kVb);
  pl->smem = 1024 + tile_smem(channel, pl->boxes, a.dim) + kTailSmem;
  if (pl->smem < 116 * 1024) pl->smem = 116 * 1024;  // one CTA per SM owns all of TMEM
  if (pl->smem > 227 * 1024) return false;
  const int64_t units = static_cast<int64_t>(a.heads) * pl->v_blocks * (n_req > 0 ? n_req : 1);
  int want = static_cast<int>(device_sm_count() / units);  // segments of the longest request that fill the GPU
  const int most = longest / (4 * kChunk);
  if (want > most) want = most;
  if (want > 16) want = 16;
  if (want < 1) want = 1;
  pl->seg_len = ceil_div(ceil_div(longest, want), kChunk) * kChunk;
  pl->segs = ceil_div(longest, pl->seg_len);
  return true;
}

// The scratch buffer, in this order (bytes, every part a multiple of 16).
struct ScratchPlan {
  int64_t factors, qk, flags, seg_state, seg_decay, start_state;
  int64_t total() const { return factors + qk + flags + seg_state + seg_decay + start_state; }
};
static ScratchPlan plan_scratch(const fr_linear_scan& a, const ChunkPlan& pl, int n_req, int n_tokens) {
  ScratchPlan s{};
  const bool channel = a.decay == FR_DECAY_CHANNEL;
  const int64_t chunks = n_tokens / kChunk + n_req + 1, per = static_cast<int64_t>(a.dim) * state_cols(a.vdim);
  s.factors = chunks * a.heads * static_cast<int64_t>(channel ? sizeof(ChannelFactors) : sizeof(HeadFactors));
  if (channel) {
    s.qk = static_cast<int64_t>(n_tokens) * a.heads * a.dim * 8;
    s.flags = (static_cast<int64_t>(n_req) * a.heads * 4 + 15) / 16 * 16;
  }
  if (pl.segs > 1) {
    s.seg_state = static_cast<int64_t>(n_req) * pl.segs * a.heads * per * 4;
    s.seg_decay = static_cast<int64_t>(n_req) * pl.segs * a.heads * a.dim * 4;
    s.start_state = static_cast<int64_t>(n_req) * a.heads * per * 4;
  }
  return s;
}

template <bool CHANNEL, bool STATE_ONLY>
static int launch_chunks(const ChunkMaps& maps, const ChunkArgs& g, int n_req, int n_segs, bool pdl, int* status, cudaStream_t stream) {
  static PerDeviceFlag f;
  if (ensure_dyn_smem(f, chunk_kernel<CHANNEL, STATE_ONLY>, 227 * 1024) != FR_OK) return FR_ERR_CUDA;
  return launch_kernel(chunk_kernel<CHANNEL, STATE_ONLY>, dim3(g.a.heads * g.pl.v_blocks, n_segs, n_req), kThreads, g.pl.smem, stream, pdl,
                       maps, g, status);
}

template <bool CHANNEL>
static int run_chunks(const ChunkArgs& g, int n_req, int longest, int n_tokens, cudaStream_t stream) {
  const fr_linear_scan& a = g.a;
  ChunkMaps m;
  const uint64_t cols = static_cast<uint64_t>(a.key_heads) * a.dim;
  int r = make_tmap_bf16_box64(&m.v, a.v, static_cast<uint64_t>(a.heads) * a.vdim, n_tokens, a.ldv, kChunk);
  if (r == FR_OK) r = make_tmap_bf16_box64(&m.out, a.out, static_cast<uint64_t>(a.heads) * a.vdim, n_tokens, a.ldo, kChunk);
  CUtensorMap* qk[4] = {&m.q, &m.q_lo, &m.k, &m.k_lo};
  for (int i = 0; i < 4 && r == FR_OK; ++i) {
    const void* p = CHANNEL ? static_cast<const void*>(g.qk + i * g.qk_stride) : (i < 2 ? a.q : a.k);
    r = make_tmap_bf16_box64(qk[i], p, cols, n_tokens, CHANNEL ? static_cast<int64_t>(cols) : (i < 2 ? a.ldq : a.ldk), kChunk);
  }
  if (r != FR_OK) return r;
  int* status = device_status_ptr();
  if (!status) return FR_ERR_CUDA;
  const bool pdl = n_tokens <= kPdlRows;
  const int chunks = ceil_div(longest, kChunk);
  if (CHANNEL) {
    const int smem = channel_smem(a);
    static PerDeviceFlag f;
    if (ensure_dyn_smem(f, channel_factor_kernel, 200 * 1024) != FR_OK) return FR_ERR_CUDA;
    if (cudaMemsetAsync(g.flags, 0, static_cast<size_t>(n_req) * a.heads * 4, stream) != cudaSuccess) return FR_ERR_CUDA;
    r = launch_kernel(channel_factor_kernel, dim3(chunks, a.heads, n_req), kPrepThreads, smem, stream, false, g);
  } else {
    r = launch_kernel(head_factor_kernel, dim3(chunks, ceil_div(a.heads, kFactorHeads), n_req), kFactorHeads * 32, 0, stream, pdl, g);
  }
  if (r == FR_OK && g.pl.segs > 1) r = launch_chunks<CHANNEL, true>(m, g, n_req, g.pl.segs - 1, pdl, status, stream);
  return r == FR_OK ? launch_chunks<CHANNEL, false>(m, g, n_req, g.pl.segs, pdl, status, stream) : r;
}

}  // namespace scan
}  // namespace fr

using namespace fr;

extern "C" int fr_linear_scan_chunks_fit(const fr_linear_scan* a) {
  scan::ChunkPlan pl;
  return a != nullptr && a->heads > 0 && a->dim > 0 && a->vdim > 0 && scan::plan_chunks(*a, 1, 1, &pl) ? 1 : 0;
}

extern "C" int64_t fr_linear_scan_chunks_scratch(const fr_linear_scan* a, int n_req, int longest, int n_tokens) {
  scan::ChunkPlan pl;
  if (a == nullptr || a->heads <= 0 || n_req <= 0 || longest <= 0 || n_tokens <= 0 || !scan::plan_chunks(*a, n_req, longest, &pl)) return -1;
  return scan::plan_scratch(*a, pl, n_req, n_tokens).total();
}

extern "C" int fr_linear_scan_chunks(const fr_linear_scan* a, int n_req, int longest, int n_tokens, int min_tokens, void* scratch,
                                     int64_t scratch_bytes, cudaStream_t stream) {
  const int st = scan::check_args(a);
  if (st != FR_OK) return st;
  FR_CHECK_ARG(n_req >= 0 && n_req <= 65535 && longest >= 0 && n_tokens >= longest);
  if (n_req == 0 || longest == 0) return FR_OK;
  scan::ChunkArgs g{};
  FR_CHECK_SUPPORTED(a->dtype == 0 && scan::plan_chunks(*a, n_req, longest, &g.pl));
  FR_CHECK_ARG(aligned16(a->q) && aligned16(a->k) && aligned16(a->v) && aligned16(a->out) && a->ldq % 8 == 0 && a->ldk % 8 == 0 &&
               a->ldv % 8 == 0 && a->ldo % 8 == 0);
  const scan::ScratchPlan sp = scan::plan_scratch(*a, g.pl, n_req, n_tokens);
  FR_CHECK_ARG(scratch && aligned16(scratch) && scratch_bytes >= sp.total());
  g.a = *a;
  g.min_tokens = min_tokens;
  uint8_t* p = static_cast<uint8_t*>(scratch);
  auto take = [&](int64_t bytes) {
    uint8_t* at = p;
    p += bytes;
    return at;
  };
  g.factors = take(sp.factors);
  g.qk = reinterpret_cast<__nv_bfloat16*>(take(sp.qk));
  g.qk_stride = sp.qk / 8;
  g.flags = reinterpret_cast<int32_t*>(take(sp.flags));
  g.seg_state = reinterpret_cast<float*>(take(sp.seg_state));
  g.seg_decay = reinterpret_cast<float*>(take(sp.seg_decay));
  g.start_state = reinterpret_cast<float*>(take(sp.start_state));
  if (a->decay == FR_DECAY_HEAD) return scan::run_chunks<false>(g, n_req, longest, n_tokens, stream);
  const int r = scan::run_chunks<true>(g, n_req, longest, n_tokens, stream);
  // what was flagged, token by token (nothing in the usual case: the CTAs look at the flag and leave)
  return r == FR_OK ? scan::rows_flagged(*a, n_req, min_tokens, g.flags, stream) : r;
}
