// bf16 prompts of the matrix-state recurrences (fr_linear_scan in the header) on tcgen05, in chunks of up to 128 tokens.
// With r_i the sum of the log decays of the chunk's tokens after its first (r_0 = 0) and S' = a_0 S the decayed old state,
// u_j the value that enters the state:
//
//     decay per head:     P_ij = e^(r_i - r_j) q_i . k_j   (j <= i)        O = e^r (Q S') + P U
//                         S <- e^(r_last) S' + K^T (e^(r_last - r_j) u_j)
//     decay per channel:  q~_i = e^(r_i) q_i,  k~_j = e^(-r_j) k_j,  P = mask(Q~ K~^T),  O = Q~ S' + P U
//                         S <- e^(r_last) (S' + K~^T U)
//
// Per channel a chunk ends early where the decays would leave the range that e^(-r) can hold, so any decays are exact
// (with a single token r is 0).
//
// Decays, factors, masks and the state are fp32. What is not bf16 to begin with (q~, k~, scaled values, P, S') enters the
// tensor cores as a sum of two bf16 numbers, 16 significant bits, in two or three products.
//
// One CTA: one head, up to 64 columns of V and S, one segment of a request. S lives in registers (thread = row of S and
// a quarter of the columns). Warps 0..15 work on operands, mask, state and output; warp 16 issues TMA and tcgen05.mma;
// warp 17 computes the next chunk's factors (decay per head). Long prompts are cut into segments that run side by side:
// a first launch finds the state that each segment adds and its total decay, the second starts every segment from the
// combination of those before it.
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
// largest -r (in powers of two) inside a chunk, per channel: e^(-r) k, its products and their sums stay far below 2^127,
// and the small halves of e^r q above 2^-126
constexpr float kMaxChannel = 86.f;

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
  const float* log2_decay;  // CHANNEL: [T, heads * dim]
  float* seg_state;    // [request, segment, head][dim][state cols]
  float* seg_decay;    // [request, segment, head][dim]
  float* start_state;  // [request, head][dim][state cols]
};

// ---------------------------------------------------------------------------
// log2 of the decays per key channel
// ---------------------------------------------------------------------------
constexpr int kDecayTokens = 32;
__global__ void __launch_bounds__(256)
log_decay_kernel(const __grid_constant__ fr_linear_scan a, int T, float* __restrict__ out) {
  extern __shared__ float s_low[];  // [tokens][rank]
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int t0 = blockIdx.x * kDecayTokens, n = min(kDecayTokens, T - t0), N = a.heads * a.dim;
  for (int e = threadIdx.x; e < n * a.rank; e += 256) s_low[e] = a.step[static_cast<int64_t>(t0 + e / a.rank) * a.ldstep + e % a.rank];
  __syncthreads();
  const int ch = blockIdx.y * 256 + threadIdx.x;
  if (ch >= N) return;
  const float* up = a.up + static_cast<int64_t>(ch) * a.rank;
  const float bias = a.step_bias[ch], f = -a.inv_tau * kLog2e;
  for (int g = 0; g < n; g += 8) {
    float z[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) z[i] = bias;
    for (int r = 0; r < a.rank; ++r) {
      const float u = up[r];
#pragma unroll
      for (int i = 0; i < 8; ++i) z[i] = fmaf(u, s_low[min(g + i, n - 1) * a.rank + r], z[i]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (g + i < n) out[static_cast<int64_t>(t0 + g + i) * N + ch] = softplus(-z[i]) * f;
  }
}

// ---------------------------------------------------------------------------
// Factors of a chunk for a decay per head, in shared memory (two sets).
struct HeadFactors {
  float r[kChunk];    // r_i (log2)
  float c[kChunk];    // log2(step_j) - r_j
  float x[kChunk];    // step_j e^(r_last - r_j)
  float first, end;   // decay of the first token, of the others
  float pad_[2];
};

// One warp, four tokens per lane.
__device__ __forceinline__ void head_factors(const fr_linear_scan& a, HeadFactors* f, int64_t t, int n, int h) {
  const int lane = threadIdx.x & 31;
  float step[4], la[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int i = lane * 4 + e;
    step[e] = i < n ? head_step(a, t + i, h) : 0.f;
  }
  const float rate = -a.rate[h] * kLog2e;
  float sum = 0.f;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    la[e] = rate * step[e];
    if (lane == 0 && e == 0) {
      f->first = ex2(la[0]);
      la[0] = 0.f;
    }
    sum += la[e];
  }
  float x = sum;
#pragma unroll
  for (int o = 1; o < 32; o *= 2) {
    const float y = __shfl_up_sync(0xffffffffu, x, o);
    if (lane >= o) x += y;
  }
  const float last = __shfl_sync(0xffffffffu, x, 31);
  float r = x - sum;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int i = lane * 4 + e;
    r += la[e];
    f->r[i] = r;
    f->c[i] = log2f(step[e]) - r;  // -inf past the end: no weight
    f->x[i] = step[e] * ex2(last - r);
  }
  if (lane == 0) f->end = ex2(last);
}

// Shared memory. HEAD: q, k tiles, two v tiles, scaled v hi and lo; CHANNEL: two v tiles, q~ hi, lo, k~ hi, lo; both: S' hi, lo.
__host__ __device__ __forceinline__ int tile_smem(bool channel, int boxes, int dim) {
  return (channel ? 2 * kBox + 4 * boxes * kBox : 2 * boxes * kBox + 4 * kBox) + 2 * dim * 128;
}
constexpr int kPartFloats = 1024;
constexpr int kTailSmem = 2 * static_cast<int>(sizeof(HeadFactors)) + (2 * kChunk + kPartFloats) * 4 + 128;

template <bool CHANNEL, bool STATE_ONLY>
__global__ void __launch_bounds__(kThreads, 1)
chunk_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
             const __grid_constant__ CUtensorMap tv, const __grid_constant__ ChunkArgs g, int* status) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const fr_linear_scan& a = g.a;
  const ChunkPlan& pl = g.pl;
  const int kq = pl.boxes * kBox;
  const uint32_t off_v = CHANNEL ? 0u : 2u * kq;                       // [2] tiles of v
  const uint32_t off_q = CHANNEL ? 2u * kBox : 0u;                     // CHANNEL: hi, lo
  const uint32_t off_k = off_q + (CHANNEL ? 2 : 1) * kq;               // CHANNEL: hi, lo
  const uint32_t off_x = off_v + 2u * kBox;                            // HEAD: scaled v hi, lo
  const uint32_t off_s = CHANNEL ? off_k + 2u * kq : off_x + 2u * kBox;
  const uint32_t s_bytes = a.dim * 128;
  HeadFactors* fac = reinterpret_cast<HeadFactors*>(smem + off_s + 2 * s_bytes);
  float* s_first = reinterpret_cast<float*>(fac + 2);  // CHANNEL: [128] decay of the chunk's first token per row of S
  float* s_end = s_first + kChunk;                     // CHANNEL: [128] decay of the others
  float* s_part = s_end + kChunk;                      // CHANNEL: partial sums of log decays
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_part + kPartFloats);
  const uint32_t bar_v = ptx::smem_u32(bars);          // [2]
  const uint32_t bar_qk = bar_v + 16, bar_g = bar_v + 24, bar_su = bar_v + 32, bar_o = bar_v + 40;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 6);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_len = reinterpret_cast<int*>(tmem_slot + 2);  // [2] CHANNEL: tokens of this chunk and the next

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool compute = tid < kCompute, issuer = tid == kCompute, factor_warp = warp == kCompute / 32 + 1;
  ptx::griddep_wait();
  const int h = blockIdx.x / pl.v_blocks, c0 = (blockIdx.x % pl.v_blocks) * kVb;
  const int b = blockIdx.z, seg = blockIdx.y;
  const int q0 = a.qo_indptr[b], q1 = a.qo_indptr[b + 1];
  const int t_begin = q0 + seg * pl.seg_len;
  if (q1 - q0 < g.min_tokens || t_begin >= q1) return;
  if (STATE_ONLY && t_begin + pl.seg_len >= q1) return;  // nothing follows the last segment
  const int t_end = min(t_begin + pl.seg_len, q1);
  const int kh = h / (a.heads / a.key_heads);
  const int vb = min(kVb, a.vdim - c0);
  const int vp = state_cols(a.vdim);

  if (tid == 0) {
    for (int i = 0; i < 6; ++i) ptx::mbar_init(bar_v + 8 * i, 1);
    *abort_flag = 0;
    s_len[0] = min(kChunk, t_end - t_begin);
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&tv);
    if (!CHANNEL) {
      ptx::prefetch_tmap(&tq);
      ptx::prefetch_tmap(&tk);
    }
  }
  if (warp == kCompute / 32) {
    __syncwarp();
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), CHANNEL ? 256 : 512);
    ptx::tmem_relinquish();
  }
  if (!CHANNEL && factor_warp) head_factors(a, fac, t_begin, min(kChunk, t_end - t_begin), h);
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  ptx::griddep_launch_dependents();  // not before the tensor memory is taken
  const uint32_t tmem = *tmem_slot;
  // scores and P (HEAD: two sets), Q S' (CHANNEL: and P U), K^T U, HEAD: P U
  const uint32_t col_in = tmem + 128, col_su = tmem + 192, col_pu = CHANNEL ? col_in : tmem + 256, col_p1 = CHANNEL ? tmem : tmem + 384;
  const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;

  auto load_v = [&](int t, int set) {  // one thread, as are the next two
    ptx::mbar_expect_tx(bar_v + 8 * set, kBox);
    ptx::tma_load_2d(base + off_v + set * kBox, &tv, h * a.vdim + c0, t, bar_v + 8 * set);
  };
  auto load_qk = [&](int t) {
    ptx::mbar_expect_tx(bar_qk, STATE_ONLY ? kq : 2 * kq);
    for (int x = 0; x < pl.boxes; ++x) {
      if (!STATE_ONLY) ptx::tma_load_2d(base + off_q + x * kBox, &tq, kh * a.dim + x * 64, t, bar_qk);
      ptx::tma_load_2d(base + off_k + x * kBox, &tk, kh * a.dim + x * 64, t, bar_qk);
    }
  };
  auto issue_scores = [&](uint32_t col) {
    constexpr uint32_t idesc = ptx::make_idesc(1u, 1u, kChunk, kChunk);
    const uint64_t qd = ptx::smem_desc_sw128(base + off_q), kd = ptx::smem_desc_sw128(base + off_k);
    const uint64_t lo = kq >> 4;
#pragma unroll 1
    for (int k = 0; k < a.dim / 16; ++k) {
      const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3);
      ptx::mma_f16(col, qd + o, kd + o, idesc, k > 0 ? 1u : 0u);
      if (CHANNEL) {
        ptx::mma_f16(col, qd + o, kd + lo + o, idesc, 1u);
        ptx::mma_f16(col, qd + lo + o, kd + o, idesc, 1u);
      }
    }
    ptx::tc_commit(bar_g);
  };
  auto wait_bar = [&](uint32_t bar, uint32_t parity, int site) {  // whole warps
    if (lane == 0) ptx::mbar_wait(bar, parity, abort_flag, status, site);
    __syncwarp();
    ptx::tc_fence_after();
  };

  // S: row of the state and a quarter of the columns
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
  // CHANNEL: a thread prepares two channels of every token of its share of the chunk
  const int pairs = a.dim / 2;
  int parts = 1;
  while (parts * 2 * pairs <= kCompute && parts < 32) parts *= 2;
  const int tp = kChunk / parts;
  const int my_part = tid / pairs, ch = 2 * (tid % pairs), i0 = my_part * tp;
  const bool prep = CHANNEL && my_part < parts;
  const int64_t ld_la = static_cast<int64_t>(a.heads) * a.dim;
  const uint32_t ch_off = (ch >> 6) * kBox + (ch & 7) * 2;  // of the channel pair in a tile of q~ or k~
  auto ch_addr = [&](int i) { return smem + off_q + ch_off + i * 128 + ((((ch & 63) >> 3) ^ (i & 7)) << 4); };

  if (issuer) {
    load_v(t_begin, 0);
    if (!CHANNEL) {
      load_qk(t_begin);
      if (!STATE_ONLY && ptx::mbar_wait(bar_qk, 0, abort_flag, status, 91)) issue_scores(tmem);
    }
  }
  __syncwarp();
  int it = 0;
  for (int t = t_begin; t < t_end; ++it) {
    const int n = min(kChunk, t_end - t);
    const int set = it & 1;
    const uint32_t set_ph = (it >> 1) & 1, ph = it & 1;
    const uint32_t col_p = CHANNEL || set == 0 ? tmem : col_p1;
    const HeadFactors* f = fac + set;
    int len = n;

    // ---- operands -----------------------------------------------------------------------------------
    if constexpr (CHANNEL) {
      const float* la = g.log2_decay + t * ld_la + h * a.dim + ch;
      if (prep) {
        float2 sum = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int i = i0; i < i0 + tp; ++i)
          if (i > 0 && i < n) {
            const float2 d = *reinterpret_cast<const float2*>(la + i * ld_la);
            sum.x += d.x;
            sum.y += d.y;
          }
        *reinterpret_cast<float2*>(s_part + my_part * a.dim + ch) = sum;
        if (my_part == 0) {
          const float2 d = *reinterpret_cast<const float2*>(la);
          *reinterpret_cast<float2*>(s_first + ch) = make_float2(ex2(d.x), ex2(d.y));
        }
      }
      __syncthreads();
      if (prep) {
        float2 r = make_float2(0.f, 0.f);
        for (int p = 0; p < my_part; ++p) {
          const float2 d = *reinterpret_cast<const float2*>(s_part + p * a.dim + ch);
          r.x += d.x;
          r.y += d.y;
        }
        const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + t * a.ldq + h * a.dim + ch;
        const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + t * a.ldk + h * a.dim + ch;
        int bad = kChunk;
        for (int g0 = i0; g0 < i0 + tp; g0 += 4) {  // four tokens' loads together (tp is a multiple of 4)
          float2 d[4];
          uint32_t kv[4], qv[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int64_t i = min(g0 + e, n - 1);
            d[e] = *reinterpret_cast<const float2*>(la + i * ld_la);
            kv[e] = *reinterpret_cast<const uint32_t*>(kp + i * a.ldk);
            if (!STATE_ONLY) qv[e] = *reinterpret_cast<const uint32_t*>(qp + i * a.ldq);
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = g0 + e;
            uint8_t* w = ch_addr(i);
            if (i < n) {
              if (i > 0) {
                r.x += d[e].x;
                r.y += d[e].y;
              }
              if (fminf(r.x, r.y) < -kMaxChannel && bad == kChunk) bad = i;
              uint32_t lo;
              if (!STATE_ONLY) {
                *reinterpret_cast<uint32_t*>(w) = split2(bf16lo(qv[e]) * a.scale * ex2(r.x), bf16hi(qv[e]) * a.scale * ex2(r.y), lo);
                *reinterpret_cast<uint32_t*>(w + kq) = lo;
              }
              *reinterpret_cast<uint32_t*>(w + 2 * kq) = split2(bf16lo(kv[e]) * ex2(-r.x), bf16hi(kv[e]) * ex2(-r.y), lo);
              *reinterpret_cast<uint32_t*>(w + 3 * kq) = lo;
              if (i == n - 1) *reinterpret_cast<float2*>(s_end + ch) = make_float2(ex2(r.x), ex2(r.y));
            } else {
              *reinterpret_cast<uint32_t*>(w + 2 * kq) = 0u;
              *reinterpret_cast<uint32_t*>(w + 3 * kq) = 0u;
            }
          }
        }
        if (bad < kChunk) atomicMin(s_len + set, bad);
      }
    }
    const float first = !compute ? 0.f : (CHANNEL ? s_first[row] : f->first);
    uint32_t xraw[8];
    if (compute) {
      if (state_thread) {
        uint8_t* dst = smem + off_s + row * 128;
#pragma unroll
        for (int c = 0; c < 16; ++c) s[c] *= first;
        if (!STATE_ONLY) {
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) hi[e] = split2(s[8 * x + 2 * e], s[8 * x + 2 * e + 1], lo[e]);
            const int o = ((quarter * 2 + x) ^ (row & 7)) << 4;
            *reinterpret_cast<uint4*>(dst + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(dst + s_bytes + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
      }
      wait_bar(bar_v + 8 * set, set_ph, 92);
      uint8_t* vrow = smem + off_v + set * kBox + row * 128;
      if constexpr (CHANNEL) {
        if (row >= n) {  // another request's values, or none
#pragma unroll
          for (int x = 0; x < 2; ++x) *reinterpret_cast<uint4*>(vrow + ((quarter * 2 + x) << 4)) = make_uint4(0, 0, 0, 0);
        }
      } else {
        const float w = f->x[row];
        const bool in = row < n;
        uint8_t* dst = smem + off_x + row * 128;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int o = ((quarter * 2 + x) ^ (row & 7)) << 4;
          uint4 v = make_uint4(0, 0, 0, 0);
          if (in) v = *reinterpret_cast<const uint4*>(vrow + o);
          else *reinterpret_cast<uint4*>(vrow + o) = v;  // another request's values, or none
          xraw[4 * x] = v.x; xraw[4 * x + 1] = v.y; xraw[4 * x + 2] = v.z; xraw[4 * x + 3] = v.w;
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) hi[e] = split2(bf16lo(xraw[4 * x + e]) * w, bf16hi(xraw[4 * x + e]) * w, lo[e]);
          *reinterpret_cast<uint4*>(dst + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(dst + kBox + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      ptx::fence_proxy_async_smem();
    }
    ptx::tc_fence_before();
    __syncthreads();
    if constexpr (CHANNEL) {
      len = s_len[set];
      if (len < n) {  // the chunk ends early: later tokens' keys leave, and the decay of the rest is another one
        if (prep) {
          for (int i = max(len, i0); i < i0 + tp; ++i) {
            uint8_t* w = ch_addr(i);
            *reinterpret_cast<uint32_t*>(w + 2 * kq) = 0u;
            *reinterpret_cast<uint32_t*>(w + 3 * kq) = 0u;
          }
        }
        if (tid < a.dim) {
          float r = 0.f;
          for (int i = 1; i < len; ++i) r += g.log2_decay[(t + i) * ld_la + h * a.dim + tid];
          s_end[tid] = ex2(r);
        }
        ptx::fence_proxy_async_smem();
        ptx::tc_fence_before();
        __syncthreads();
      }
    }
    const int next = t + len;
    const int k_tok = (len + 15) / 16;  // steps of 16 tokens
    if (issuer) {
      ptx::tc_fence_after();
      const uint32_t idesc_o = ptx::make_idesc(1u, 1u, kChunk, vb) | (1u << 16);  // B is MN-major
      const uint32_t idesc_s = idesc_o | (1u << 15);                              // A too
      if (CHANNEL) {
        if (next < t_end) load_v(next, set ^ 1);
        if (!STATE_ONLY) issue_scores(col_p);
      }
      if (!STATE_ONLY) {
        const uint64_t qd = ptx::smem_desc_sw128(base + off_q), qlo = qd + (kq >> 4);
        const uint64_t sd = ptx::smem_desc_sw128(base + off_s), slo = sd + (s_bytes >> 4);  // 64 columns: no leading offset
#pragma unroll 1
        for (int k = 0; k < a.dim / 16; ++k) {
          const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3), so = k * 128u;
          ptx::mma_f16(col_in, qd + o, sd + so, idesc_o, k > 0 ? 1u : 0u);
          ptx::mma_f16(col_in, qd + o, slo + so, idesc_o, 1u);
          if (CHANNEL) ptx::mma_f16(col_in, qlo + o, sd + so, idesc_o, 1u);
        }
      } else if (!CHANNEL) {
        ptx::mbar_wait(bar_qk, ph, abort_flag, status, 96);
      }
      // A = K^T: rows of S by tokens, a second box of rows for more than 64 (else the first once more, unused)
      const uint64_t lead = static_cast<uint64_t>(((pl.boxes > 1 ? kBox : 0) >> 4) & 0x3fff) << 16;
      const uint64_t kt = (ptx::smem_desc_sw128(base + off_k) & ~(static_cast<uint64_t>(0x3fffu) << 16)) | lead;
      const uint64_t ud = ptx::smem_desc_sw128(base + (CHANNEL ? off_v + set * kBox : off_x));
#pragma unroll 1
      for (int k = 0; k < k_tok; ++k) {
        const uint64_t o = k * 128u;
        ptx::mma_f16(col_su, kt + o, ud + o, idesc_s, k > 0 ? 1u : 0u);
        ptx::mma_f16(col_su, CHANNEL ? kt + (kq >> 4) + o : kt + o, CHANNEL ? ud + o : ud + kBox / 16 + o, idesc_s, 1u);
      }
      ptx::tc_commit(bar_su);
      if (!CHANNEL && next < t_end) {  // the other v tile is free, those of q and k are with these products
        load_v(next, set ^ 1);
        if (ptx::mbar_wait(bar_su, ph, abort_flag, status, 97)) load_qk(next);
      }
    }
    if (!CHANNEL && factor_warp && next < t_end) head_factors(a, fac + (set ^ 1), next, min(kChunk, t_end - next), h);
    __syncwarp();

    // ---- P as two bf16 halves over the scores, 32 columns per thread: [16 hi | 16 lo] ------------------
    if (!STATE_ONLY) {
      if (compute) {
        wait_bar(bar_g, ph, 93);
        if (quarter * 32 < len) {
          uint32_t p[32];
          if (quarter > (warp & 3)) {  // keys after every query of this warp
#pragma unroll
            for (int c = 0; c < 32; ++c) p[c] = 0u;
          } else {
            uint32_t gv[32];
            ptx::tmem_ld_32x32(col_p + lane_off + quarter * 32, gv);
            const float ri = CHANNEL ? 0.f : f->r[row];
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
      __syncthreads();
      if (issuer) {
        ptx::tc_fence_after();
        const uint32_t idesc_o = ptx::make_idesc(1u, 1u, kChunk, vb) | (1u << 16);
        const uint64_t vd = ptx::smem_desc_sw128(base + off_v + set * kBox);
#pragma unroll 1
        for (int k = 0; k < k_tok; ++k) {
          const uint32_t pc = col_p + (k >> 1) * 32 + (k & 1) * 8;
          ptx::mma_f16_ts(col_pu, pc, vd + k * 128u, idesc_o, CHANNEL || k > 0 ? 1u : 0u);
          ptx::mma_f16_ts(col_pu, pc + 16, vd + k * 128u, idesc_o, 1u);
        }
        ptx::tc_commit(bar_o);
        if (!CHANNEL && next < t_end && ptx::mbar_wait(bar_qk, ph ^ 1u, abort_flag, status, 98)) issue_scores(set == 0 ? col_p1 : tmem);
      }
      __syncwarp();
    }

    // ---- new state, output ---------------------------------------------------------------------------
    if (compute) {
      wait_bar(bar_su, ph, 94);
      uint32_t v[16];
      ptx::tmem_ld_32x16(col_su + lane_off + col0, v);
      ptx::tmem_ld_wait();
      if (state_thread) {
        const float end = CHANNEL ? s_end[row] : f->end;
#pragma unroll
        for (int c = 0; c < 16; ++c)
          s[c] = CHANNEL ? end * (s[c] + __uint_as_float(v[c])) : fmaf(end, s[c], __uint_as_float(v[c]));
        decay_all *= first * end;
      }
      if (!STATE_ONLY) {
        uint32_t y[16];
        if (!CHANNEL) ptx::tmem_ld_32x16(col_in + lane_off + col0, y);
        wait_bar(bar_o, ph, 95);
        ptx::tmem_ld_32x16(col_pu + lane_off + col0, v);
        ptx::tmem_ld_wait();
        if (row < len && my_cols) {
          __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (t + row) * a.ldo + h * a.vdim + c0 + col0;
          const float er = CHANNEL ? 0.f : ex2(f->r[row]);
          uint32_t w[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            float y0 = __uint_as_float(v[2 * e]), y1 = __uint_as_float(v[2 * e + 1]);
            if (!CHANNEL) {
              y0 = fmaf(skip, bf16lo(xraw[e]), a.scale * fmaf(er, __uint_as_float(y[2 * e]), y0));
              y1 = fmaf(skip, bf16hi(xraw[e]), a.scale * fmaf(er, __uint_as_float(y[2 * e + 1]), y1));
            }
            w[e] = pack_bf16(y0, y1);
          }
          *reinterpret_cast<uint4*>(out) = make_uint4(w[0], w[1], w[2], w[3]);
          *reinterpret_cast<uint4*>(out + 8) = make_uint4(w[4], w[5], w[6], w[7]);
        }
        __syncwarp();
      }
      ptx::tc_fence_before();
    }
    if (CHANNEL && issuer) s_len[set ^ 1] = min(kChunk, t_end - next);
    __syncthreads();
    ptx::tc_fence_after();
    if (*abort_flag) break;
    t = next;
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
  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == kCompute / 32) {
    ptx::tc_fence_after();
    ptx::tmem_dealloc(tmem, CHANNEL ? 256 : 512);
  }
}

// ---------------------------------------------------------------------------
static bool plan_chunks(const fr_linear_scan& a, int n_req, int longest, ChunkPlan* pl) {
  if (a.dim % 16 != 0 || a.vdim % 16 != 0 || a.dim > kChunk) return false;
  const bool channel = a.decay == FR_DECAY_CHANNEL;
  pl->boxes = (a.dim + 63) / 64;
  pl->v_blocks = ceil_div(a.vdim, kVb);
  pl->smem = 1024 + tile_smem(channel, pl->boxes, a.dim) + kTailSmem;
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
static int64_t state_scratch(const fr_linear_scan& a, const ChunkPlan& pl, int n_req) {
  if (pl.segs <= 1) return 0;
  const int64_t per = static_cast<int64_t>(a.dim) * state_cols(a.vdim);
  return static_cast<int64_t>(n_req) * a.heads * (pl.segs * (per + a.dim) + per) * 4;
}
static int64_t decay_scratch(const fr_linear_scan& a, int n_tokens) {
  return a.decay == FR_DECAY_CHANNEL ? static_cast<int64_t>(n_tokens) * a.heads * a.dim * 4 : 0;
}

template <bool CHANNEL, bool STATE_ONLY>
static int launch_chunks(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const ChunkArgs& g, int n_req, int n_segs,
                         bool pdl, int* status, cudaStream_t stream) {
  static PerDeviceFlag f;
  if (ensure_dyn_smem(f, chunk_kernel<CHANNEL, STATE_ONLY>, 227 * 1024) != FR_OK) return FR_ERR_CUDA;
  return launch_kernel(chunk_kernel<CHANNEL, STATE_ONLY>, dim3(g.a.heads * g.pl.v_blocks, n_segs, n_req), kThreads, g.pl.smem, stream, pdl,
                       tq, tk, tv, g, status);
}

template <bool CHANNEL>
static int run_chunks(const ChunkArgs& g, int n_req, int n_tokens, cudaStream_t stream) {
  const fr_linear_scan& a = g.a;
  CUtensorMap tq, tk, tv;
  int r = make_tmap_bf16_box64(&tv, a.v, static_cast<uint64_t>(a.heads) * a.vdim, n_tokens, a.ldv, kChunk);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tq, a.q, static_cast<uint64_t>(a.key_heads) * a.dim, n_tokens, a.ldq, kChunk);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tk, a.k, static_cast<uint64_t>(a.key_heads) * a.dim, n_tokens, a.ldk, kChunk);
  if (r != FR_OK) return r;
  int* status = device_status_ptr();
  if (!status) return FR_ERR_CUDA;
  const bool pdl = n_tokens <= kPdlRows;
  if (g.pl.segs > 1) {
    r = launch_chunks<CHANNEL, true>(tq, tk, tv, g, n_req, g.pl.segs - 1, pdl, status, stream);
    if (r != FR_OK) return r;
  }
  return launch_chunks<CHANNEL, false>(tq, tk, tv, g, n_req, g.pl.segs, pdl, status, stream);
}

}  // namespace scan
}  // namespace fr

using namespace fr;

extern "C" int fr_linear_scan_chunks_fit(int decay, int dim, int vdim) {
  fr_linear_scan a{};
  a.decay = decay;
  a.heads = 1;
  a.dim = dim;
  a.vdim = vdim;
  scan::ChunkPlan pl;
  return dim > 0 && vdim > 0 && scan::plan_chunks(a, 1, 1, &pl) ? 1 : 0;
}

extern "C" int64_t fr_linear_scan_chunks_scratch(const fr_linear_scan* a, int n_req, int longest, int n_tokens) {
  scan::ChunkPlan pl;
  if (a == nullptr || a->heads <= 0 || n_req <= 0 || longest <= 0 || n_tokens <= 0 || !scan::plan_chunks(*a, n_req, longest, &pl)) return -1;
  return scan::decay_scratch(*a, n_tokens) + scan::state_scratch(*a, pl, n_req) + 16;
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
  FR_CHECK_ARG(scratch && aligned16(scratch) && scratch_bytes >= fr_linear_scan_chunks_scratch(a, n_req, longest, n_tokens));
  g.a = *a;
  g.min_tokens = min_tokens;
  float* p = static_cast<float*>(scratch);
  if (a->decay == FR_DECAY_CHANNEL) {
    const int smem = scan::kDecayTokens * a->rank * 4;
    FR_CHECK_SUPPORTED(smem <= 48 * 1024);
    g.log2_decay = p;
    const int r = launch_kernel(scan::log_decay_kernel, dim3(ceil_div(n_tokens, scan::kDecayTokens), ceil_div(a->heads * a->dim, 256)), 256,
                                smem, stream, n_tokens <= kPdlRows, *a, n_tokens, p);
    if (r != FR_OK) return r;
    p += scan::decay_scratch(*a, n_tokens) / 4;
  }
  const int64_t per = static_cast<int64_t>(a->dim) * scan::state_cols(a->vdim);
  g.seg_state = p;
  g.start_state = p + static_cast<int64_t>(n_req) * a->heads * g.pl.segs * per;
  g.seg_decay = g.start_state + static_cast<int64_t>(n_req) * a->heads * per;
  return a->decay == FR_DECAY_CHANNEL ? scan::run_chunks<true>(g, n_req, n_tokens, stream) : scan::run_chunks<false>(g, n_req, n_tokens, stream);
}
