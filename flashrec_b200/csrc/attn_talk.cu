// Talking heads for bf16 prompts (the TALK side of fr_mix_attn_tc with scratch). Every output head mixes all H softmax
// maps, and an SM's tensor memory cannot hold the accumulators of all heads, so a kernel that keeps its maps on chip
// has to recompute them for every v head. Here the maps are computed once, in blocks of token tiles:
//   1. talk_maps_kernel   (tile, head): one pass over the keys; writes fp32 exponentials E_h [128, keys] relative to
//                         a running row maximum and, per 32 keys, the factor that turns them into weights
//   2. talk_mix_kernel    M_h = sum_g T[h, g] factor_g E_g in fp32, written as bf16 (the MMA operand)
//   3. talk_values_kernel (tile, head): O_h = M_h V, a plain tcgen05 product with V as it lies in the cache
// Scratch per tile: H x 128 x keys x (4 + 2 + 1/8) bytes.
#include "attn_mix.cuh"

namespace fr {
namespace talk {

using mix::kLog2e;
using mix::kM;
using mix::kTileN;

constexpr int kThreads = 192;

// Keys a tile of up to 128 tokens may span, rounded to whole pages.
static int tile_keys(const fr_mix_attn& a, int max_pos) {
  const int64_t all = (static_cast<int64_t>(max_pos) + kTileN) / kTileN * kTileN;
  const int64_t span = (static_cast<int64_t>(a.mask_size) + 127 + 126 + kTileN - 1) / kTileN * kTileN;
  return static_cast<int>(all < span ? all : span);
}

// ---------------------------------------------------------------------------
// 1. maps. warp 0 = TMA, warp 1 = MMA, warps 2..9 = two threads per token, 32 keys of a tile each (own running maximum;
//    they meet at the end). S has four TMEM buffers, so the product
//    runs up to three key tiles ahead of the softmax threads.
// ---------------------------------------------------------------------------
constexpr int kSBufs = 4;
constexpr int kKStages = 3;
constexpr int kMapThreads = 64 + 8 * 32;
constexpr int kFactorKeys = 32;  // keys that share a factor

__global__ void __launch_bounds__(kMapThreads, 2)
talk_maps_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
                 const __grid_constant__ fr_mix_attn a, int boxes, const int32_t* __restrict__ tiles, float* __restrict__ maps,
                 float* __restrict__ factors, int ldp, int* status) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const int q_bytes = boxes * kM * 128, k_bytes = boxes * kTileN * 128;
  const uint32_t sm_q = base, sm_k = base + q_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + q_bytes + kKStages * k_bytes);
  const uint32_t bar_q = ptx::smem_u32(bars);
  const uint32_t bar_kfull = bar_q + 8, bar_kempty = bar_kfull + 8 * kKStages;
  const uint32_t bar_sfull = bar_kempty + 8 * kKStages, bar_sempty = bar_sfull + 8 * kSBufs;
  const uint32_t bar_pair = bar_sempty + 8 * kSBufs;  // [4] a warp and its partner
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5 + 2 * kKStages + 2 * kSBufs);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* pages = reinterpret_cast<int*>(bars + 32);
  float2* pair_buf = reinterpret_cast<float2*>(pages + mix::kPageList);  // [2 halves][128 rows] maximum, sum
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int head = blockIdx.y, kvh = head / (a.heads / a.kv_heads);
  const int req = tiles[3 * blockIdx.x], row0 = tiles[3 * blockIdx.x + 1], n_tok = tiles[3 * blockIdx.x + 2];
  const int pos0 = static_cast<int>(a.pos[row0]);
  const int32_t* table = a.req_to_token + a.req_rows[req] * a.table_stride;
  const mix::KeyTiles kt = mix::key_tiles(a, pos0, pos0 + n_tok - 1);
  const int total = kt.n;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    ptx::mbar_init(bar_q, 1);
    for (int i = 0; i < kKStages; ++i) {
      ptx::mbar_init(bar_kfull + 8 * i, 1);
      ptx::mbar_init(bar_kempty + 8 * i, 1);
    }
    for (int i = 0; i < kSBufs; ++i) {
      ptx::mbar_init(bar_sfull + 8 * i, 1);
      ptx::mbar_init(bar_sempty + 8 * i, 8);
    }
    for (int i = 0; i < 4; ++i) ptx::mbar_init(bar_pair + 8 * i, 2);
    *abort_flag = 0;
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&tq);
    ptx::prefetch_tmap(&tk);
  }
  mix::load_pages(a, table, kt, pages);
  if (warp == 1) {
    __syncwarp();
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), kSBufs * kTileN);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      ptx::mbar_expect_tx(bar_q, q_bytes);
      for (int b = 0; b < boxes; ++b) ptx::tma_load_2d(sm_q + b * kM * 128, &tq, head * a.dim + b * 64, row0, bar_q);
      bool ok = true;
      for (int it = 0; it < total && ok; ++it) {
        const int st = it % kKStages;
        ok = ptx::mbar_wait(bar_kempty + 8 * st, ((it / kKStages) & 1) ^ 1u, abort_flag, status, 91);
        if (!ok) break;
        ptx::mbar_expect_tx(bar_kfull + 8 * st, k_bytes);
        const int row = mix::page_at(a, table, kt, pages, it);
        for (int b = 0; b < boxes; ++b)
          ptx::tma_load_2d(sm_k + st * k_bytes + b * kTileN * 128, &tk, kvh * a.dim + b * 64, row, bar_kfull + 8 * st);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = ptx::make_idesc(1u, 1u, kM, kTileN);
      bool ok = ptx::mbar_wait(bar_q, 0, abort_flag, status, 92);
      for (int it = 0; it < total && ok; ++it) {
        const int st = it % kKStages, sb = it % kSBufs;
        ok = ptx::mbar_wait(bar_sempty + 8 * sb, ((it / kSBufs) & 1) ^ 1u, abort_flag, status, 93) &&
             ptx::mbar_wait(bar_kfull + 8 * st, (it / kKStages) & 1, abort_flag, status, 94);
        if (!ok) break;
        ptx::tc_fence_after();
        for (int k = 0; k < a.dim / 16; ++k)
          ptx::mma_f16(tmem_base + sb * kTileN, ptx::smem_desc_sw128(sm_q + (k >> 2) * kM * 128) + 2u * (k & 3),
                       ptx::smem_desc_sw128(sm_k + st * k_bytes + (k >> 2) * kTileN * 128) + 2u * (k & 3), idesc,
                       k > 0 ? 1u : 0u);
        ptx::tc_commit(bar_kempty + 8 * st);
        ptx::tc_commit(bar_sfull + 8 * sb);
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3, half = (warp - 2) >> 2, r = quad * 32 + lane;
    const int i = pos0 + min(r, n_tok - 1);
    const int lo = static_cast<int>(mix::lowest_key(a, i));
    const int keep = a.mask == FR_MASK_CHUNK ? 0 : a.keep_first;
    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    const float scale = a.scale * kLog2e;
    const float slope = a.slopes != nullptr ? a.slopes[head] * kLog2e : 0.f;
    float* out = maps + ((static_cast<int64_t>(blockIdx.x) * a.heads + head) * kM + r) * ldp + half * kFactorKeys;
    float* fac = factors + ((static_cast<int64_t>(blockIdx.x) * a.heads + head) * (ldp / kFactorKeys) + half) * kM + r;
    auto wait_all = [&](uint32_t bar, uint32_t parity, int site) -> bool {
      int okw = 0;
      if (lane == 0) okw = ptx::mbar_wait(bar, parity, abort_flag, status, site) ? 1 : 0;
      okw = __shfl_sync(0xffffffffu, okw, 0);
      __syncwarp();
      return okw != 0;
    };
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int it = 0; it < total; ++it) {
      const int sb = it % kSBufs;
      ok = wait_all(bar_sfull + 8 * sb, (it / kSBufs) & 1, 95);
      if (!ok) break;
      ptx::tc_fence_after();
      uint32_t sv[32];
      ptx::tmem_ld_32x32(tmem_base + lane_off + sb * kTileN + half * kFactorKeys, sv);
      ptx::tmem_ld_wait();
      ptx::tc_fence_before();
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(bar_sempty + 8 * sb);
      const int j0 = kt.at(it) * kTileN + half * kFactorKeys;
      const float bias0 = slope * static_cast<float>(j0 - i);
#pragma unroll
      for (int c = 0; c < 32; ++c)
        sv[c] = __float_as_uint(fmaf(__uint_as_float(sv[c]), scale, fmaf(slope, static_cast<float>(c), bias0)));
      if (__any_sync(0xffffffffu, j0 + 31 > i || (j0 < lo && j0 + 32 > keep))) {
        const uint32_t vis = static_cast<uint32_t>(mix::visible_bits(j0, i, lo, keep));
#pragma unroll
        for (int c = 0; c < 32; ++c)
          if (!((vis >> c) & 1u)) sv[c] = 0xff800000u;  // -inf
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 32; ++c) mx[c & 3] = fmaxf(mx[c & 3], __uint_as_float(sv[c]));
      const float mn = fmaxf(m, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));
      if (mn > m) {
        l *= mix::ex2(m - mn);
        m = mn;
      }
      const float ref = m == -INFINITY ? 0.f : m;
      float ps[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        uint32_t w[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float p = mix::ex2(__uint_as_float(sv[8 * x + e]) - ref);
          ps[e & 3] += p;
          w[e] = __float_as_uint(p);
        }
        ptx::st_global_v8(out + it * kTileN + 8 * x, w);
      }
      l += (ps[0] + ps[1]) + (ps[2] + ps[3]);
      fac[it * 2 * kM] = m;
    }
    if (ok) {
      pair_buf[half * kM + r] = make_float2(m, l);
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(bar_pair + 8 * quad);
      ok = wait_all(bar_pair + 8 * quad, 0, 99);
    }
    if (ok) {
      const float2 other = pair_buf[(half ^ 1) * kM + r];
      const float mt = fmaxf(m, other.x);  // finite: a token sees itself
      const float inv = 1.0f / (l * mix::ex2(m - mt) + other.y * mix::ex2(other.x - mt));
      for (int j = 0; j < total; ++j) fac[j * 2 * kM] = mix::ex2(fac[j * 2 * kM] - mt) * inv;  // 0 where nothing was visible yet
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
    ptx::tmem_dealloc(tmem_base, kSBufs * kTileN);
  }
}

// ---------------------------------------------------------------------------
// 2. M_h = sum_g T[h, g] factor_g E_g. A thread holds four keys of one row for kHeadBlock output heads; the products
//    run two to an instruction.
// ---------------------------------------------------------------------------
constexpr int kHeadBlock = 16;

constexpr int kMixThreads = 128;
constexpr int kMixAhead = 8;  // maps on their way while as many are used

__global__ void __launch_bounds__(kMixThreads, 3)
talk_mix_kernel(const __grid_constant__ fr_mix_attn a, const int32_t* __restrict__ tiles, const float* __restrict__ maps,
                const float* __restrict__ factors, __nv_bfloat16* __restrict__ mixed, int ldp) {
  extern __shared__ uint64_t coef[];  // [heads (source)][kHeadBlock], every value twice
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int tile = blockIdx.y, h0 = blockIdx.z * kHeadBlock;
  const int row0 = tiles[3 * tile + 1], n_tok = tiles[3 * tile + 2];
  const int pos0 = static_cast<int>(a.pos[row0]);
  const int keys = mix::key_tiles(a, pos0, pos0 + n_tok - 1).n * kTileN;
  const int quads = keys / 4;
  if (static_cast<int>(blockIdx.x) * kMixThreads >= kM * quads) return;
  for (int e = threadIdx.x; e < a.heads * kHeadBlock; e += kMixThreads) {
    const int g = e / kHeadBlock, h = h0 + e % kHeadBlock;
    const float t = h < a.heads ? a.coef[static_cast<int64_t>(h) * a.heads + g] : 0.f;
    coef[e] = mix::pack_f32x2(t, t);
  }
  __syncthreads();
  const int64_t head_stride = static_cast<int64_t>(kM) * ldp;
  const int64_t fac_stride = static_cast<int64_t>(ldp / kFactorKeys) * kM;
  for (int e = blockIdx.x * kMixThreads + threadIdx.x; e < kM * quads; e += gridDim.x * kMixThreads) {
    const int r = e / quads, c = e % quads * 4;
    const int64_t off = (static_cast<int64_t>(tile) * a.heads * kM + r) * ldp + c;
    const float* fac = factors + static_cast<int64_t>(tile) * a.heads * fac_stride + (c / kFactorKeys) * kM + r;
    uint64_t acc[kHeadBlock][2] = {};
    float4 nxt[kMixAhead];
    float nf[kMixAhead];
#pragma unroll
    for (int x = 0; x < kMixAhead; ++x) {
      nxt[x] = make_float4(0, 0, 0, 0);
      nf[x] = 0.f;
      if (x < a.heads) {
        nxt[x] = __ldcs(reinterpret_cast<const float4*>(maps + off + x * head_stride));
        nf[x] = __ldg(fac + x * fac_stride);
      }
    }
    for (int g0 = 0; g0 < a.heads; g0 += kMixAhead) {
      uint64_t p[kMixAhead][2];
#pragma unroll
      for (int x = 0; x < kMixAhead; ++x) {
        p[x][0] = mix::pack_f32x2(nxt[x].x * nf[x], nxt[x].y * nf[x]);
        p[x][1] = mix::pack_f32x2(nxt[x].z * nf[x], nxt[x].w * nf[x]);
      }
#pragma unroll
      for (int x = 0; x < kMixAhead; ++x) {
        if (g0 + kMixAhead + x < a.heads) {  // the next maps are on their way while these are used
          nxt[x] = __ldcs(reinterpret_cast<const float4*>(maps + off + (g0 + kMixAhead + x) * head_stride));
          nf[x] = __ldg(fac + (g0 + kMixAhead + x) * fac_stride);
        }
      }
#pragma unroll
      for (int x = 0; x < kMixAhead; ++x) {
        if (g0 + x < a.heads) {
          const uint64_t* cf = coef + (g0 + x) * kHeadBlock;
#pragma unroll
          for (int h = 0; h < kHeadBlock; h += 2) {
            const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(cf + h);
            acc[h][0] = mix::fma_f32x2(t.x, p[x][0], acc[h][0]);
            acc[h][1] = mix::fma_f32x2(t.x, p[x][1], acc[h][1]);
            acc[h + 1][0] = mix::fma_f32x2(t.y, p[x][0], acc[h + 1][0]);
            acc[h + 1][1] = mix::fma_f32x2(t.y, p[x][1], acc[h + 1][1]);
          }
        }
      }
    }
#pragma unroll
    for (int h = 0; h < kHeadBlock; ++h)
      if (h0 + h < a.heads) {
        float f[4];
        mix::unpack_f32x2(acc[h][0], f[0], f[1]);
        mix::unpack_f32x2(acc[h][1], f[2], f[3]);
        *reinterpret_cast<uint2*>(mixed + off + (h0 + h) * head_stride) =
            make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
      }
  }
}

// ---------------------------------------------------------------------------
// 3. O_h = M_h V: M by TMA from the scratch (K-major), V by TMA from the cache pages (MN-major)
// ---------------------------------------------------------------------------
constexpr int kStages = 3;

__global__ void __launch_bounds__(kThreads, 2)
talk_values_kernel(const __grid_constant__ CUtensorMap tm, const __grid_constant__ CUtensorMap tv,
                   const __grid_constant__ fr_mix_attn a, int v_boxes, int v_cols, int tmem_cols,
                   const int32_t* __restrict__ tiles, int* status) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const int m_bytes = kM * 128, v_bytes = v_boxes * kTileN * 128, stage = m_bytes + v_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kStages * stage);
  const uint32_t bar_full = ptx::smem_u32(bars), bar_empty = bar_full + 8 * kStages, bar_done = bar_empty + 8 * kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * kStages + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* pages = reinterpret_cast<int*>(bars + 32);
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int head = blockIdx.y, vh = head / (a.heads / a.kv_heads);
  const int req = tiles[3 * blockIdx.x], row0 = tiles[3 * blockIdx.x + 1], n_tok = tiles[3 * blockIdx.x + 2];
  const int pos0 = static_cast<int>(a.pos[row0]);
  const int32_t* table = a.req_to_token + a.req_rows[req] * a.table_stride;
  const mix::KeyTiles kt = mix::key_tiles(a, pos0, pos0 + n_tok - 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kStages; ++i) {
      ptx::mbar_init(bar_full + 8 * i, 1);
      ptx::mbar_init(bar_empty + 8 * i, 1);
    }
    ptx::mbar_init(bar_done, 1);
    *abort_flag = 0;
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&tm);
    ptx::prefetch_tmap(&tv);
  }
  mix::load_pages(a, table, kt, pages);
  if (warp == 1) {
    __syncwarp();
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), tmem_cols);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      for (int it = 0; it < kt.n && ok; ++it) {
        const int st = it % kStages;
        ok = ptx::mbar_wait(bar_empty + 8 * st, ((it / kStages) & 1) ^ 1u, abort_flag, status, 96);
        if (!ok) break;
        ptx::mbar_expect_tx(bar_full + 8 * st, stage);
        ptx::tma_load_2d(base + st * stage, &tm, it * kTileN, (static_cast<int>(blockIdx.x) * a.heads + head) * kM, bar_full + 8 * st);
        const int row = mix::page_at(a, table, kt, pages, it);
        for (int b = 0; b < v_boxes; ++b)
          ptx::tma_load_2d(base + st * stage + m_bytes + b * kTileN * 128, &tv, vh * a.vdim + b * 64, row, bar_full + 8 * st);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = ptx::make_idesc(1u, 1u, kM, a.vdim) | (1u << 16);  // B is MN-major
      bool ok = true;
      for (int it = 0; it < kt.n && ok; ++it) {
        const int st = it % kStages;
        ok = ptx::mbar_wait(bar_full + 8 * st, (it / kStages) & 1, abort_flag, status, 97);
        if (!ok) break;
        ptx::tc_fence_after();
        const uint64_t m_desc = ptx::smem_desc_sw128(base + st * stage);
        const uint64_t v_desc = mix::smem_desc_mn(base + st * stage + m_bytes, kTileN * 128);
        for (int k = 0; k < kTileN / 16; ++k)
          ptx::mma_f16(tmem_base, m_desc + 2u * k, v_desc + static_cast<uint64_t>(k * 16 * 128 >> 4), idesc,
                       (it | k) != 0 ? 1u : 0u);
        ptx::tc_commit(bar_empty + 8 * st);
        if (it + 1 == kt.n) ptx::tc_commit(bar_done);
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3, r = quad * 32 + lane;
    int okw = 0;
    if (lane == 0) okw = ptx::mbar_wait(bar_done, 0, abort_flag, status, 98) ? 1 : 0;
    okw = __shfl_sync(0xffffffffu, okw, 0);
    ptx::tc_fence_after();
    if (okw) {
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + (row0 + min(r, n_tok - 1)) * a.ldo +
                           static_cast<int64_t>(head) * a.vdim;
#pragma unroll 1
      for (int c = 0; c < v_cols / 32; ++c) {
        uint32_t o[32];
        ptx::tmem_ld_32x32(tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + c * 32, o);
        ptx::tmem_ld_wait();
        if (r < n_tok) {
          uint4* d4 = reinterpret_cast<uint4*>(dst + c * 32);
#pragma unroll
          for (int x = 0; x < 4; ++x)
            if (c * 32 + x * 8 < a.vdim)
              d4[x] = make_uint4(pack_bf16(__uint_as_float(o[8 * x]), __uint_as_float(o[8 * x + 1])),
                                 pack_bf16(__uint_as_float(o[8 * x + 2]), __uint_as_float(o[8 * x + 3])),
                                 pack_bf16(__uint_as_float(o[8 * x + 4]), __uint_as_float(o[8 * x + 5])),
                                 pack_bf16(__uint_as_float(o[8 * x + 6]), __uint_as_float(o[8 * x + 7])));
        }
        __syncwarp();
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
    ptx::tmem_dealloc(tmem_base, tmem_cols);
  }
}

}  // namespace talk

int64_t talk_tc_tile_bytes(const fr_mix_attn& a, int max_pos) {
  return static_cast<int64_t>(a.heads) * talk::kM * (talk::tile_keys(a, max_pos) / 8 * 49);  // E, M, factors
}

int talk_tc(const fr_mix_attn& a, const int32_t* tiles, int n_tiles, int n_rows, int max_pos, void* scratch,
            int64_t scratch_bytes, cudaStream_t stream) {
  using namespace talk;
  const int ldp = tile_keys(a, max_pos);
  const int64_t per_tile = talk_tc_tile_bytes(a, max_pos);
  int block = static_cast<int>(scratch_bytes / per_tile < n_tiles ? scratch_bytes / per_tile : n_tiles);
  if (block < 1) return FR_ERR_BAD_ARG;
  if (block > 32768 / a.heads) block = 32768 / a.heads;
  float* maps = static_cast<float*>(scratch);
  const int64_t values = static_cast<int64_t>(block) * a.heads * kM * ldp;
  float* factors = maps + values;
  __nv_bfloat16* mixed = reinterpret_cast<__nv_bfloat16*>(factors + values / kFactorKeys);
  const int boxes = (a.dim + 63) / 64, v_boxes = (a.vdim + 63) / 64, v_cols = (a.vdim + 31) / 32 * 32;
  int tmem_cols = 32;
  while (tmem_cols < v_cols) tmem_cols *= 2;
  const int smem_maps = 1024 + boxes * (kM + kKStages * kTileN) * 128 + 256 + mix::kPageList * 4 + 2 * kM * 8;
  const int smem_values = 1024 + kStages * (kM + v_boxes * kTileN) * 128 + 256 + mix::kPageList * 4;
  const int smem_mix = a.heads * kHeadBlock * 8;
  FR_CHECK_SUPPORTED(smem_mix <= 48 * 1024 && smem_maps <= 227 * 1024 && smem_values <= 227 * 1024);
  static PerDeviceFlag f0, f1;
  if (ensure_dyn_smem(f0, talk_maps_kernel, 227 * 1024) != FR_OK) return FR_ERR_CUDA;
  if (ensure_dyn_smem(f1, talk_values_kernel, 227 * 1024) != FR_OK) return FR_ERR_CUDA;
  CUtensorMap tq, tk, tv, tm;
  int r = make_tmap_bf16_box64(&tq, a.q, static_cast<uint64_t>(a.heads) * a.dim, n_rows, a.ldq, kM);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tk, a.k, static_cast<uint64_t>(a.kv_heads) * a.dim, a.num_slots, a.ldk, kTileN);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tv, a.v, static_cast<uint64_t>(a.kv_heads) * a.vdim, a.num_slots, a.ldv, kTileN);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tm, mixed, ldp, static_cast<uint64_t>(block) * a.heads * kM, ldp, kM);
  if (r != FR_OK) return r;
  int* status = device_status_ptr();
  if (!status) return FR_ERR_CUDA;
  const bool pdl = n_rows <= kPdlRows;
  for (int t0 = 0; t0 < n_tiles; t0 += block) {
    const int n = n_tiles - t0 < block ? n_tiles - t0 : block;
    const int32_t* tl = tiles + 3 * static_cast<int64_t>(t0);
    r = launch_kernel(talk_maps_kernel, dim3(n, a.heads), kMapThreads, smem_maps, stream, pdl, tq, tk, a, boxes, tl, maps,
                      factors, ldp, status);
    if (r == FR_OK)
      r = launch_kernel(talk_mix_kernel, dim3(ceil_div(static_cast<int64_t>(kM) * ldp / 4, kMixThreads), n, ceil_div(a.heads, kHeadBlock)), kMixThreads,
                        smem_mix, stream, pdl, a, tl, maps, factors, mixed, ldp);
    if (r == FR_OK)
      r = launch_kernel(talk_values_kernel, dim3(n, a.heads), kThreads, smem_values, stream, pdl, tm, tv, a, v_boxes, v_cols, tmem_cols,
                        tl, status);
    if (r != FR_OK) return r;
  }
  return FR_OK;
}

}  // namespace fr
