// bf16 prompts of the matrix-state recurrences (fr_linear_scan in the header) on tcgen05, in chunks of up to 128 tokens.
// With r_i the sum of the log decays of the chunk's tokens after its first (r_0 = 0) and S' = a_0 S the decayed old state,
//
//     q~_i = e^(r_i) q_i,   k~_j = e^(-r_j) k_j,   P = mask(Q~ K~^T)      (j <= i)
//     O = Q~ S' + P V,      S <- e^(r_last) (S' + K~^T V)
//
// For a decay per head the factors are one number per token: Q and K stay as they are, V is scaled instead and the rows
// of O at the end. A chunk ends early where the decays would leave the range that e^(-r) can hold, so any decays are
// exact; with a single token r is 0.
//
// Decays, factors, masks and the state are fp32. What is not bf16 to begin with (q~, k~, scaled v, P, S') enters the
// tensor cores as a sum of two bf16 numbers, 16 significant bits, in two or three products.
//
// One CTA: one head, up to 64 columns of V and S, one segment of a request. S lives in registers (thread = row of S and
// half of the columns). Long prompts are cut into segments that run side by side: a first launch finds the state that
// each segment adds and its total decay, the second starts every segment from the combination of those before it.
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
constexpr int kCompute = 256;          // threads of the compute warps
constexpr int kThreads = kCompute + 32;
constexpr float kLog2e = 1.4426950408889634f;
// largest -r (in powers of two) inside a chunk: e^(-r) v, its products and their sums stay below 2^127; per channel the
// small side is a pair of bf16 numbers too and must stay above 2^-126
constexpr float kMaxHead = 96.f, kMaxChannel = 86.f;

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
  int tile_bytes;  // one set of TMA tiles
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
  // two sets of TMA tiles (HEAD: q, k, v; CHANNEL: v), then
  // CHANNEL: q~ hi, lo, k~ hi, lo;  HEAD: low halves of the scaled v;  both: S' hi, lo
  const uint32_t off_work = 2 * pl.tile_bytes;
  const uint32_t off_s = off_work + (CHANNEL ? 4 * kq : kBox);
  const uint32_t s_bytes = a.dim * 128;
  const uint32_t off_f = (off_s + 2 * s_bytes + 15) & ~15u;
  float* s_first = reinterpret_cast<float*>(smem + off_f);  // [128] decay of the chunk's first token, per row of S
  float* s_end = s_first + 128;                             // [128] decay of the others
  float* s_row = s_end + 128;                               // [128] HEAD: e^(r_i)
  float* s_w = s_row + 128;                                 // [128] HEAD: step * e^(-r_i)
  float* s_part = s_w + 128;                                // [512] partial sums of log decays
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_part + 512);
  const uint32_t bar_tile = ptx::smem_u32(bars);            // [2]
  const uint32_t bar_g = bar_tile + 16, bar_su = bar_tile + 24, bar_o = bar_tile + 32;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_len = reinterpret_cast<int*>(tmem_slot + 2);       // tokens of the chunk

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
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
    for (int i = 0; i < 5; ++i) ptx::mbar_init(bar_tile + 8 * i, 1);
    *abort_flag = 0;
    *s_len = min(kChunk, t_end - t_begin);
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&tv);
    if (!CHANNEL) {
      ptx::prefetch_tmap(&tq);
      ptx::prefetch_tmap(&tk);
    }
  }
  if (warp == 8) {
    __syncwarp();
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), 256);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  ptx::griddep_launch_dependents();  // not before the tensor memory is taken
  const uint32_t tmem = *tmem_slot;
  const uint32_t col_p = tmem, col_o = tmem + 128, col_su = tmem + 192;
  const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;

  auto load_tiles = [&](int t, int set) {  // one thread
    const uint32_t dst = base + set * pl.tile_bytes, bar = bar_tile + 8 * set;
    ptx::mbar_expect_tx(bar, pl.tile_bytes - (!CHANNEL && STATE_ONLY ? kq : 0));
    uint32_t o = dst;
    if (!CHANNEL) {
      for (int x = 0; x < pl.boxes; ++x, o += kBox)
        if (!STATE_ONLY) ptx::tma_load_2d(o, &tq, kh * a.dim + x * 64, t, bar);
      for (int x = 0; x < pl.boxes; ++x, o += kBox) ptx::tma_load_2d(o, &tk, kh * a.dim + x * 64, t, bar);
    }
    ptx::tma_load_2d(o, &tv, h * a.vdim + c0, t, bar);
  };
  auto wait_bar = [&](uint32_t bar, uint32_t parity, int site) {  // whole warps
    if (lane == 0) ptx::mbar_wait(bar, parity, abort_flag, status, site);
    __syncwarp();
    ptx::tc_fence_after();
  };

  // S: row of the state and half of the columns
  const int row = tid & 127, half = (tid >> 7) & 1;
  const bool state_thread = tid < kCompute && row < a.dim;
  float s[32];
  float decay_all = 1.0f;
  {
    const int64_t per = static_cast<int64_t>(a.dim) * vp;
    const int64_t here = static_cast<int64_t>(row) * vp + c0 + half * 32;
    const int64_t seg0 = static_cast<int64_t>(b) * pl.segs;
#pragma unroll
    for (int c = 0; c < 32; ++c) s[c] = 0.f;
    auto columns = [&](auto&& f) {
#pragma unroll
      for (int c = 0; c < 32; c += 4)
        if (half * 32 + c < vb) f(c);
    };
    if (state_thread) {
      if (seg == 0) {
        const bool fresh = a.pos[q0] == 0;
        const bool saved = !STATE_ONLY && pl.segs > 1 && q1 - q0 > pl.seg_len;
        const float* src = saved ? g.start_state + (static_cast<int64_t>(b) * a.heads + h) * per
                                 : a.state + (a.state_slots[b] * a.heads + h) * per;
        columns([&](int c) {
          float4 v = make_float4(0, 0, 0, 0);
          if (saved || !fresh) v = *reinterpret_cast<const float4*>(src + here + c);
          s[c] = v.x; s[c + 1] = v.y; s[c + 2] = v.z; s[c + 3] = v.w;
          if (STATE_ONLY)
            *reinterpret_cast<float4*>(g.start_state + (static_cast<int64_t>(b) * a.heads + h) * per + here + c) = v;
        });
      } else if (!STATE_ONLY) {
        for (int r = 0; r < seg; ++r) {
          const int64_t id = (seg0 + r) * a.heads + h;
          const float d = r == 0 ? 0.f : g.seg_decay[id * a.dim + row];
          columns([&](int c) {
            const float4 v = *reinterpret_cast<const float4*>(g.seg_state + id * per + here + c);
            s[c] = fmaf(d, s[c], v.x); s[c + 1] = fmaf(d, s[c + 1], v.y);
            s[c + 2] = fmaf(d, s[c + 2], v.z); s[c + 3] = fmaf(d, s[c + 3], v.w);
          });
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
  const int my_pair = tid % pairs, my_part = tid / pairs;
  const bool prep = CHANNEL && tid < kCompute && my_part < parts;

  if (tid == kCompute) load_tiles(t_begin, 0);
  __syncwarp();
  int it = 0;
  for (int t = t_begin; t < t_end; ++it) {
    const int n = min(kChunk, t_end - t);
    const int set = it & 1;
    const uint32_t set_ph = (it >> 1) & 1, ph = it & 1;
    const uint32_t tiles = base + set * pl.tile_bytes;
    const uint32_t a_q = CHANNEL ? base + off_work : tiles, a_k = CHANNEL ? a_q + 2 * kq : tiles + kq;
    const uint32_t a_v = CHANNEL ? tiles : tiles + 2 * kq, a_vlo = base + off_work;
    const uint32_t a_s = base + off_s;

    // ---- factors of the chunk -----------------------------------------------------------------------
    if constexpr (CHANNEL) {
      const int64_t ld = static_cast<int64_t>(a.heads) * a.dim;
      const float* la = g.log2_decay + t * ld + h * a.dim + 2 * my_pair;
      const int i0 = my_part * tp;
      if (prep) {
        float2 sum = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int i = i0; i < i0 + tp; ++i)
          if (i > 0 && i < n) {
            const float2 d = *reinterpret_cast<const float2*>(la + i * ld);
            sum.x += d.x;
            sum.y += d.y;
          }
        *reinterpret_cast<float2*>(s_part + my_part * a.dim + 2 * my_pair) = sum;
        if (my_part == 0) {
          const float2 d = *reinterpret_cast<const float2*>(la);
          s_first[2 * my_pair] = ex2(d.x);
          s_first[2 * my_pair + 1] = ex2(d.y);
        }
      }
      __syncthreads();
      if (prep) {
        float2 r = make_float2(0.f, 0.f);
        for (int p = 0; p < my_part; ++p) {
          const float2 d = *reinterpret_cast<const float2*>(s_part + p * a.dim + 2 * my_pair);
          r.x += d.x;
          r.y += d.y;
        }
        const int ch = 2 * my_pair;
        const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + t * a.ldq + h * a.dim + ch;
        const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + t * a.ldk + h * a.dim + ch;
        const uint32_t col = (ch >> 6) * kBox + (ch & 7) * 2;
        const int chunk16 = (ch & 63) >> 3;
        int bad = kChunk;
#pragma unroll 4
        for (int i = i0; i < i0 + tp; ++i) {
          const uint32_t dst = col + i * 128 + ((chunk16 ^ (i & 7)) << 4);
          uint8_t* w = smem + off_work + dst;
          if (i < n) {
            if (i > 0) {
              const float2 d = *reinterpret_cast<const float2*>(la + i * ld);
              r.x += d.x;
              r.y += d.y;
            }
            if ((r.x < -kMaxChannel || r.y < -kMaxChannel) && bad == kChunk) bad = i;
            const uint32_t kv = *reinterpret_cast<const uint32_t*>(kp + i * a.ldk);
            uint32_t lo;
            if (!STATE_ONLY) {
              const uint32_t qv = *reinterpret_cast<const uint32_t*>(qp + i * a.ldq);
              const uint32_t qh = split2(bf16lo(qv) * a.scale * ex2(r.x), bf16hi(qv) * a.scale * ex2(r.y), lo);
              *reinterpret_cast<uint32_t*>(w) = qh;
              *reinterpret_cast<uint32_t*>(w + kq) = lo;
            }
            const uint32_t khi = split2(bf16lo(kv) * ex2(-r.x), bf16hi(kv) * ex2(-r.y), lo);
            *reinterpret_cast<uint32_t*>(w + 2 * kq) = khi;
            *reinterpret_cast<uint32_t*>(w + 3 * kq) = lo;
            if (i == n - 1) {
              s_end[ch] = ex2(r.x);
              s_end[ch + 1] = ex2(r.y);
            }
          } else {
            *reinterpret_cast<uint32_t*>(w + 2 * kq) = 0u;
            *reinterpret_cast<uint32_t*>(w + 3 * kq) = 0u;
          }
        }
        if (bad < kChunk) atomicMin(s_len, bad);
      }
    } else {
      float x = 0.f, step = 0.f;
      if (warp < 4) {
        if (tid < n) step = head_step(a, t + tid, h);
        const float la = -a.rate[h] * step * kLog2e;
        if (tid == 0) *s_first = ex2(la);
        x = tid == 0 ? 0.f : la;
#pragma unroll
        for (int o = 1; o < 32; o *= 2) {
          const float y = __shfl_up_sync(0xffffffffu, x, o);
          if (lane >= o) x += y;
        }
        if (lane == 31) s_part[warp] = x;
      }
      __syncthreads();
      if (warp < 4) {
        for (int w = 0; w < warp; ++w) x += s_part[w];
        if (tid < n && x < -kMaxHead) atomicMin(s_len, tid);
        s_row[tid] = ex2(x);
        s_w[tid] = step * ex2(-x);
      }
    }
    __syncthreads();
    const int len = *s_len, next = t + len;

    // ---- operands -----------------------------------------------------------------------------------
    if (tid == kCompute) {
      if (next < t_end) load_tiles(next, set ^ 1);
      if (!CHANNEL && !STATE_ONLY && ptx::mbar_wait(bar_tile + 8 * set, set_ph, abort_flag, status, 91)) {
        constexpr uint32_t idesc = ptx::make_idesc(1u, 1u, kChunk, kChunk);
        const uint64_t qd = ptx::smem_desc_sw128(a_q), kd = ptx::smem_desc_sw128(a_k);
        for (int k = 0; k < a.dim / 16; ++k) {
          const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3);
          ptx::mma_f16(col_p, qd + o, kd + o, idesc, k > 0 ? 1u : 0u);
        }
        ptx::tc_commit(bar_g);
      }
    }
    __syncwarp();
    uint32_t xraw[16];
    float first = 0.f;
    if (tid < kCompute) {
      if (state_thread) {
        first = s_first[CHANNEL ? row : 0];
        uint8_t* dst = smem + off_s + row * 128;
#pragma unroll
        for (int c = 0; c < 32; ++c) s[c] *= first;
        if (!STATE_ONLY) {
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) hi[e] = split2(s[8 * x + 2 * e], s[8 * x + 2 * e + 1], lo[e]);
            const int o = ((half * 4 + x) ^ (row & 7)) << 4;
            *reinterpret_cast<uint4*>(dst + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(dst + s_bytes + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
      }
      wait_bar(bar_tile + 8 * set, set_ph, 92);
      uint8_t* vrow = smem + (a_v - base) + row * 128;
      if constexpr (CHANNEL) {
        if (len < n) {  // the chunk ends early: later tokens' keys leave, and the last token's decay is another one
          if (prep) {
            const int ch = 2 * my_pair;
            for (int i = max(len, my_part * tp); i < (my_part + 1) * tp; ++i) {
              uint8_t* w = smem + off_work + (ch >> 6) * kBox + (ch & 7) * 2 + i * 128 + ((((ch & 63) >> 3) ^ (i & 7)) << 4);
              *reinterpret_cast<uint32_t*>(w + 2 * kq) = 0u;
              *reinterpret_cast<uint32_t*>(w + 3 * kq) = 0u;
            }
          }
          if (tid < a.dim) {
            const int64_t ld = static_cast<int64_t>(a.heads) * a.dim;
            float r = 0.f;
            for (int i = 1; i < len; ++i) r += g.log2_decay[(t + i) * ld + h * a.dim + tid];
            s_end[tid] = ex2(r);
          }
        }
        if (row >= n) {  // another request's values, or none
#pragma unroll
          for (int x = 0; x < 4; ++x) *reinterpret_cast<uint4*>(vrow + ((half * 4 + x) << 4)) = make_uint4(0, 0, 0, 0);
        }
      } else {
        const float w = s_w[row];
        const bool in = row < len;
        uint8_t* lrow = smem + (a_vlo - base) + row * 128;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int o = ((half * 4 + x) ^ (row & 7)) << 4;
          const uint4 v = *reinterpret_cast<const uint4*>(vrow + o);
          xraw[4 * x] = v.x; xraw[4 * x + 1] = v.y; xraw[4 * x + 2] = v.z; xraw[4 * x + 3] = v.w;
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e)
            hi[e] = split2(in ? bf16lo(xraw[4 * x + e]) * w : 0.f, in ? bf16hi(xraw[4 * x + e]) * w : 0.f, lo[e]);
          *reinterpret_cast<uint4*>(vrow + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(lrow + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      ptx::fence_proxy_async_smem();
    }
    ptx::tc_fence_before();
    __syncthreads();
    const int k_tok = (len + 15) / 16;  // steps of 16 tokens
    if (tid == kCompute) {
      ptx::tc_fence_after();
      constexpr uint32_t idesc_g = ptx::make_idesc(1u, 1u, kChunk, kChunk);
      const uint32_t idesc_o = ptx::make_idesc(1u, 1u, kChunk, vb) | (1u << 16);  // B is MN-major
      const uint32_t idesc_s = idesc_o | (1u << 15);                              // A too
      if (!STATE_ONLY) {
        const uint64_t qd = ptx::smem_desc_sw128(a_q), kd = ptx::smem_desc_sw128(a_k);
        const uint64_t qlo = qd + (kq >> 4), klo = kd + (kq >> 4);
        if (CHANNEL) {
          for (int k = 0; k < a.dim / 16; ++k) {
            const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3);
            ptx::mma_f16(col_p, qd + o, kd + o, idesc_g, k > 0 ? 1u : 0u);
            ptx::mma_f16(col_p, qd + o, klo + o, idesc_g, 1u);
            ptx::mma_f16(col_p, qlo + o, kd + o, idesc_g, 1u);
          }
          ptx::tc_commit(bar_g);
        }
        const uint64_t sd = ptx::smem_desc_sw128(a_s), slo = sd + (s_bytes >> 4);  // 64 columns: no leading offset
        for (int k = 0; k < a.dim / 16; ++k) {
          const uint64_t o = (k >> 2) * (kBox / 16) + 2u * (k & 3), so = k * 128u;
          ptx::mma_f16(col_o, qd + o, sd + so, idesc_o, k > 0 ? 1u : 0u);
          ptx::mma_f16(col_o, qd + o, slo + so, idesc_o, 1u);
          if (CHANNEL) ptx::mma_f16(col_o, qlo + o, sd + so, idesc_o, 1u);
        }
      }
      // A = K~^T: rows of S by tokens, a second box of rows for more than 64 (else the first once more, unused)
      const uint64_t lead = static_cast<uint64_t>(((pl.boxes > 1 ? kBox : 0) >> 4) & 0x3fff) << 16;
      const uint64_t kt = (ptx::smem_desc_sw128(a_k) & ~(static_cast<uint64_t>(0x3fffu) << 16)) | lead, ktlo = kt + (kq >> 4);
      const uint64_t vd = ptx::smem_desc_sw128(a_v), vlo = ptx::smem_desc_sw128(a_vlo);
      for (int k = 0; k < k_tok; ++k) {
        const uint64_t o = k * 128u;
        ptx::mma_f16(col_su, kt + o, vd + o, idesc_s, k > 0 ? 1u : 0u);
        ptx::mma_f16(col_su, CHANNEL ? ktlo + o : kt + o, CHANNEL ? vd + o : vlo + o, idesc_s, 1u);
      }
      ptx::tc_commit(bar_su);
    }
    __syncwarp();

    // ---- mask; P as two bf16 halves over the scores --------------------------------------------------
    if (!STATE_ONLY) {
      uint32_t hi[32], lo[32];
      if (tid < kCompute) {
        wait_bar(bar_g, ph, 93);
        if (half * 64 < len) {
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            uint32_t gv[32];
            ptx::tmem_ld_32x32(col_p + lane_off + half * 64 + x * 32, gv);
            ptx::tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 16; ++c) {
              const int j = half * 64 + x * 32 + 2 * c;
              hi[x * 16 + c] = split2(j <= row ? __uint_as_float(gv[2 * c]) : 0.f, j + 1 <= row ? __uint_as_float(gv[2 * c + 1]) : 0.f,
                                      lo[x * 16 + c]);
            }
          }
        }
        ptx::tc_fence_before();
      }
      __syncthreads();
      if (tid < kCompute) {
        ptx::tc_fence_after();
        if (half * 64 < len) {
          ptx::tmem_st_32x32(col_p + lane_off + half * 32, hi);
          ptx::tmem_st_32x32(col_p + lane_off + 64 + half * 32, lo);
          ptx::tmem_st_wait();
        }
        ptx::tc_fence_before();
      }
      __syncthreads();
      if (tid == kCompute) {
        ptx::tc_fence_after();
        const uint32_t idesc_o = ptx::make_idesc(1u, 1u, kChunk, vb) | (1u << 16);
        const uint64_t vd = ptx::smem_desc_sw128(a_v), vlo = ptx::smem_desc_sw128(a_vlo);
        for (int k = 0; k < k_tok; ++k) {
          const uint64_t o = k * 128u;
          ptx::mma_f16_ts(col_o, col_p + 8u * k, vd + o, idesc_o, 1u);
          ptx::mma_f16_ts(col_o, col_p + 64 + 8u * k, vd + o, idesc_o, 1u);
          if (!CHANNEL) ptx::mma_f16_ts(col_o, col_p + 8u * k, vlo + o, idesc_o, 1u);
        }
        ptx::tc_commit(bar_o);
      }
      __syncwarp();
    }

    // ---- new state, output ---------------------------------------------------------------------------
    if (tid < kCompute) {
      wait_bar(bar_su, ph, 94);
      uint32_t v[32];
      ptx::tmem_ld_32x32(col_su + lane_off + half * 32, v);
      ptx::tmem_ld_wait();
      if (state_thread) {
        const float end = CHANNEL ? s_end[row] : s_row[len - 1];
#pragma unroll
        for (int c = 0; c < 32; ++c) s[c] = end * (s[c] + __uint_as_float(v[c]));
        decay_all *= first * end;
      }
      if (!STATE_ONLY) {
        wait_bar(bar_o, ph, 95);
        ptx::tmem_ld_32x32(col_o + lane_off + half * 32, v);
        ptx::tmem_ld_wait();
        if (row < len) {
          __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (t + row) * a.ldo + h * a.vdim + c0 + half * 32;
          const float f = CHANNEL ? 1.0f : s_row[row] * a.scale;
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float y0 = __uint_as_float(v[8 * x + 2 * e]) * f, y1 = __uint_as_float(v[8 * x + 2 * e + 1]) * f;
              if (!CHANNEL) {
                y0 = fmaf(skip, bf16lo(xraw[4 * x + e]), y0);
                y1 = fmaf(skip, bf16hi(xraw[4 * x + e]), y1);
              }
              w[e] = pack_bf16(y0, y1);
            }
            if (half * 32 + x * 8 < vb) *reinterpret_cast<uint4*>(out + x * 8) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
        __syncwarp();
      }
      ptx::tc_fence_before();
    }
    if (tid == kCompute) *s_len = min(kChunk, t_end - next);
    __syncthreads();
    ptx::tc_fence_after();
    if (*abort_flag) break;
    t = next;
  }

  if (state_thread) {
    const int64_t per = static_cast<int64_t>(a.dim) * vp;
    float* dst = nullptr;
    if (STATE_ONLY) {
      const int64_t id = (static_cast<int64_t>(b) * pl.segs + seg) * a.heads + h;
      dst = g.seg_state + id * per;
      if (half == 0 && c0 == 0) g.seg_decay[id * a.dim + row] = decay_all;
    } else if (t_end == q1) {
      dst = a.state + (a.state_slots[b] * a.heads + h) * per;
    }
    if (dst != nullptr) {
#pragma unroll
      for (int c = 0; c < 32; c += 4)
        if (half * 32 + c < vb)
          *reinterpret_cast<float4*>(dst + static_cast<int64_t>(row) * vp + c0 + half * 32 + c) = make_float4(s[c], s[c + 1], s[c + 2], s[c + 3]);
    }
  }
  ptx::tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 8) {
    ptx::tc_fence_after();
    ptx::tmem_dealloc(tmem, 256);
  }
}

// ---------------------------------------------------------------------------
static bool plan_chunks(const fr_linear_scan& a, int n_req, int longest, ChunkPlan* pl) {
  if (a.dim % 16 != 0 || a.vdim % 16 != 0 || a.dim > kChunk) return false;
  const bool channel = a.decay == FR_DECAY_CHANNEL;
  pl->boxes = (a.dim + 63) / 64;
  pl->v_blocks = ceil_div(a.vdim, kVb);
  pl->tile_bytes = channel ? kBox : (2 * pl->boxes + 1) * kBox;
  pl->smem = 1024 + 2 * pl->tile_bytes + (channel ? 4 * pl->boxes * kBox : kBox) + 2 * a.dim * 128 + 16 + (4 * 128 + 512) * 4 + 64;
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
