// Helpers shared by the mixed-map attention kernels (attn_mix.cu, attn_talk.cu).
#pragma once

#include "fr_common.cuh"
#include "sm100_ptx.cuh"

namespace fr {

int* device_status_ptr();  // capi.cu
int make_tmap_bf16_box64(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, int64_t pitch,
                         uint32_t box_rows);  // dense_proj.cu

namespace mix {

constexpr float kLog2e = 1.4426950408889634f;

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
template <typename T>
__device__ __forceinline__ void st_f(T* p, float v) { *p = v; }
template <>
__device__ __forceinline__ void st_f<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Visible keys of the query at position i: [0, n_first) and [lo, i].
struct Visible {
  int64_t lo;
  int n_first, n;
  __device__ __forceinline__ int64_t key(int idx) const { return idx < n_first ? idx : lo + (idx - n_first); }
};
__device__ __forceinline__ int64_t lowest_key(const fr_mix_attn& a, int64_t i) {
  if (a.mask == FR_MASK_CHUNK) return i / a.mask_size * a.mask_size;
  return i - a.mask_size + 1 > 0 ? i - a.mask_size + 1 : 0;
}
__device__ __forceinline__ Visible visible_keys(const fr_mix_attn& a, int64_t i, int max_keys) {
  Visible v;
  v.lo = lowest_key(a, i);
  v.n_first = a.mask == FR_MASK_CHUNK ? 0 : static_cast<int>(a.keep_first < v.lo ? a.keep_first : v.lo);
  const int64_t n = v.n_first + (i - v.lo + 1);
  v.n = static_cast<int>(n < max_keys ? n : max_keys);
  return v;
}
__device__ __forceinline__ int64_t slot_of(const fr_mix_attn& a, int64_t table_row, int64_t j) {
  const int64_t s = a.req_to_token[table_row * a.table_stride + j];
  return s < 0 ? 0 : (s >= a.num_slots ? a.num_slots - 1 : s);
}
// i-th source map that reads k head kh
__device__ __forceinline__ int source_of(const fr_mix_attn& a, int kh, int i) {
  const int rep = a.heads / a.kv_heads;
  return a.mix == FR_MIX_DIFF ? 2 * ((kh >> 1) * rep + i) + (kh & 1) : kh * rep + i;
}

constexpr int kM = 128;     // tokens per tensor-core tile (UMMA M)
constexpr int kTileN = 64;  // keys per tile: one cache page

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
// two fp32 operations per instruction
__device__ __forceinline__ uint64_t pack_f32x2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpack_f32x2(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t add_f32x2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// Bit c: the query at i, whose window or chunk begins at lo, sees the key j0 + c.
__device__ __forceinline__ uint64_t low_bits(int n) { return n <= 0 ? 0ull : (n >= 64 ? ~0ull : (1ull << n) - 1ull); }
__device__ __forceinline__ uint64_t visible_bits(int j0, int i, int lo, int keep) {
  return low_bits(i - j0 + 1) & (~low_bits(lo - j0) | low_bits(keep - j0));
}

// MN-major operand tile as TMA writes it with the 128-byte swizzle: rows of 64 values (128 bytes), one row per k;
// 8-row groups 1024 bytes apart (stride), 64-value column blocks `lead` bytes apart (leading offset).
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr, uint32_t lead) {
  uint64_t d = ptx::smem_desc_sw128(addr) & ~(static_cast<uint64_t>(0x3fffu) << 16);
  return d | static_cast<uint64_t>((lead >> 4) & 0x3fffu) << 16;
}

// Key tiles of up to 128 consecutive tokens [pos0, pos_last]: [0, n_keep) hold kept first tokens, from t_lo on the rest.
struct KeyTiles {
  int n_keep, t_lo, n;
  __device__ __forceinline__ int at(int jj) const { return jj < n_keep ? jj : t_lo + jj - n_keep; }
};
__device__ __forceinline__ KeyTiles key_tiles(const fr_mix_attn& a, int pos0, int pos_last) {
  KeyTiles k;
  k.t_lo = static_cast<int>(lowest_key(a, pos0)) / kTileN;
  k.n_keep = a.mask == FR_MASK_CHUNK ? 0 : min((min(a.keep_first, pos_last + 1) + kTileN - 1) / kTileN, k.t_lo);
  k.n = k.n_keep + pos_last / kTileN - k.t_lo + 1;
  return k;
}
// First of the 64 consecutive slots of a key page (clamped: a bad table entry reads a wrong page, not outside memory).
__device__ __forceinline__ int page_row(const fr_mix_attn& a, const int32_t* table, int tile) {
  const int s = table[static_cast<int64_t>(tile) * kTileN];
  const int last = static_cast<int>(a.num_slots) - kTileN;
  return s < 0 ? 0 : (s > last ? last : s);
}

// The tiles' page rows, read once by all threads (before a __syncthreads) so that the TMA producer does not wait for
// a table entry per tile.
constexpr int kPageList = 512;
__device__ __forceinline__ void load_pages(const fr_mix_attn& a, const int32_t* table, const KeyTiles& kt, int* pages) {
  for (int j = threadIdx.x; j < kt.n && j < kPageList; j += blockDim.x) pages[j] = page_row(a, table, kt.at(j));
}
__device__ __forceinline__ int page_at(const fr_mix_attn& a, const int32_t* table, const KeyTiles& kt, const int* pages, int j) {
  return j < kPageList ? pages[j] : page_row(a, table, kt.at(j));
}

}  // namespace mix
}  // namespace fr
