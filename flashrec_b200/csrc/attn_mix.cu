// Attention whose outputs are linear combinations of several softmax maps over the same values
// (fr_mix_attn in the header): differential attention (two maps per head, weights 1 and -lambda, the result
// divided by its root mean square), talking heads (all heads' maps, one matrix row per output head) and ordinary
// attention (one map per head, optionally times a sigmoid per head), with
// a sliding window that keeps the first tokens or with chunks, and an optional linear distance bias.
//
// Because the mixture is linear, sum_s coef[o, s] (P_s V) = (sum_s coef[o, s] P_s) V:
//   * mix_scores_kernel + mix_values_kernel (fr_mix_attn_rows: decode, f32, any head size) write the scores of
//     every visible key, mix the normalised weights and pass over V once; keys may be split over CTAs;
//   * mix_tc_kernel (fr_mix_attn_tc: bf16 prompts, tcgen05) runs one flash pass per source map and adds
//     coef[o, s] / l_s times its result to the outputs' accumulators, which stay in TMEM beside S and O.
#include "attn_mix.cuh"

namespace fr {

int talk_tc(const fr_mix_attn& a, const int32_t* tiles, int n_tiles, int n_rows, int max_pos, void* scratch,
            int64_t scratch_bytes, cudaStream_t stream);  // attn_talk.cu
int64_t talk_tc_tile_bytes(const fr_mix_attn& a, int max_pos);

namespace mix {

constexpr int kKeyBlock = 64;
constexpr int kMaxPer = 4;  // key blocks per CTA of the scores kernel when the batch fills the GPU anyway

// ---------------------------------------------------------------------------
// scores of one row, one k head and `per` blocks of 64 keys for every source map that reads that k head; per block and map the
// maximum and the sum of exponentials
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
mix_scores_kernel(const __grid_constant__ fr_mix_attn a, int row0, int max_keys, int n_blocks, int per,
                  float* __restrict__ scores, float2* __restrict__ stats) {
  extern __shared__ float sm[];
  const int rep = a.heads / a.kv_heads;
  const int n_src = a.mix == FR_MIX_DIFF ? 2 * a.heads : a.heads;
  float* qs = sm;                       // [rep][dim]
  float* sc = sm + rep * a.dim;         // [rep][64 per]
  __shared__ int64_t slots[kMaxPer * kKeyBlock];
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int lrow = blockIdx.z, kh = blockIdx.y, blk = blockIdx.x;
  const int64_t t = row0 + lrow;
  const int64_t i = a.pos[t];
  const Visible vis = visible_keys(a, i, max_keys);
  const int span = per * kKeyBlock;
  const int k0 = blk * span;
  if (k0 >= vis.n) return;
  const int nk = min(span, vis.n - k0);
  const T* q = static_cast<const T*>(a.q) + t * a.ldq;
  for (int e = threadIdx.x; e < rep * (a.dim / 8); e += 128) {
    const int s = e / (a.dim / 8), c = e % (a.dim / 8) * 8;
    float v[8];
    load8<T>(q + static_cast<int64_t>(source_of(a, kh, s)) * a.dim + c, v);
#pragma unroll
    for (int x = 0; x < 8; ++x) qs[s * a.dim + c + x] = v[x];
  }
  const int64_t table_row = a.req_rows[a.tok_req[t]];
  for (int e = threadIdx.x; e < nk; e += 128) slots[e] = slot_of(a, table_row, vis.key(k0 + e));
  __syncthreads();
  int lanes = 1;  // lanes per key
  while (lanes < 32 && lanes * 8 < a.dim) lanes *= 2;
  const int lane_k = threadIdx.x % lanes;
  const T* kc = static_cast<const T*>(a.k) + static_cast<int64_t>(kh) * a.dim;
  const int keys_at_once = 128 / lanes;
  const bool one_chunk = lanes * 8 >= a.dim;  // a lane holds its share of a key in registers
  const bool in_dim = lane_k * 8 < a.dim;
  // groups of up to four keys per thread, their rows in flight together; trip counts are CTA-uniform (the shuffles
  // are whole-warp)
  for (int kb = 0; kb < span; kb += 4 * keys_at_once) {
    float kv[4][8] = {};
    const T* kr[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int kk = kb + x * keys_at_once + threadIdx.x / lanes;
      kr[x] = kc + slots[min(kk, nk - 1)] * a.ldk;
      if (one_chunk && in_dim && kk < nk) load8<T>(kr[x] + lane_k * 8, kv[x]);
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      if (kb + x * keys_at_once >= span) break;
      const int kk = kb + x * keys_at_once + threadIdx.x / lanes;
      const bool live = kk < nk;
      const float dist = static_cast<float>(i - vis.key(k0 + (live ? kk : 0)));
      for (int s = 0; s < rep; ++s) {
        const float* qr = qs + s * a.dim;
        float acc = 0.f;
        if (one_chunk) {
          if (in_dim) {
            const float4 q0 = *reinterpret_cast<const float4*>(qr + lane_k * 8);
            const float4 q1 = *reinterpret_cast<const float4*>(qr + lane_k * 8 + 4);
            acc = kv[x][0] * q0.x + kv[x][1] * q0.y + kv[x][2] * q0.z + kv[x][3] * q0.w + kv[x][4] * q1.x + kv[x][5] * q1.y +
                  kv[x][6] * q1.z + kv[x][7] * q1.w;
          }
        } else {
          for (int c = lane_k * 8; c < a.dim; c += lanes * 8) {
            float v[8];
            load8<T>(kr[x] + c, v);
#pragma unroll
            for (int y = 0; y < 8; ++y) acc = fmaf(v[y], qr[c + y], acc);
          }
        }
        for (int o = lanes / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane_k == 0 && kk < span) {
          float v = acc * a.scale;
          if (a.slopes != nullptr) v -= a.slopes[source_of(a, kh, s)] * dist;
          sc[s * span + kk] = live ? v : -INFINITY;
        }
      }
    }
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = warp; e < rep * per; e += 4) {  // (map, block of 64)
    const int s = e / per, sub = e % per, c0 = sub * kKeyBlock;
    if (c0 >= nk) continue;
    const int64_t row = static_cast<int64_t>(lrow) * n_src + source_of(a, kh, s);
    const float v0 = sc[s * span + c0 + lane], v1 = sc[s * span + c0 + 32 + lane];
    const float m = warp_max(fmaxf(v0, v1));
    const float l = warp_sum(expf(v0 - m) + expf(v1 - m));
    const int k1 = k0 + c0;
    if (k1 + lane < max_keys) scores[row * max_keys + k1 + lane] = v0;
    if (k1 + 32 + lane < max_keys) scores[row * max_keys + k1 + 32 + lane] = v1;
    if (lane == 0) stats[row * n_blocks + blk * per + sub] = make_float2(m, l);
  }
}

// ---------------------------------------------------------------------------
// mixture of the maps and product with V for one row, one kv head and one share of the keys
// ---------------------------------------------------------------------------
constexpr int kValThreads = 256;
constexpr int kValKeys = 256;  // keys per pass (weights of all maps in shared memory)

// sigmoid(head_gate) of one output head, 1 without a gate
__device__ __forceinline__ float head_gate_of(const fr_mix_attn& a, int64_t t, int head) {
  return a.head_gate != nullptr ? 1.0f / (1.0f + expf(-a.head_gate[t * a.ld_gate + head])) : 1.0f;
}

// Root-mean-square scaling (DIFF) or head gate, and store of one output head; f [vdim] in shared memory.
template <typename T>
__device__ __forceinline__ void finish_head(const fr_mix_attn& a, int64_t t, int head, const float* f, float* red) {
  float r = 1.0f;
  if (a.mix == FR_MIX_DIFF) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.vdim; c += kValThreads) ss += f[c] * f[c];  // padded columns hold zero
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < kValThreads / 32; ++w) tot += red[w];
    r = a.out_scale / sqrtf(tot / static_cast<float>(a.vdim_true) + a.eps);
    __syncthreads();
  } else {
    r = head_gate_of(a, t, head);
  }
  T* out = static_cast<T*>(a.out) + t * a.ldo + static_cast<int64_t>(head) * a.vdim;
  for (int c = threadIdx.x; c < a.vdim; c += kValThreads) st_f(out + c, f[c] * r);
}

// OB: output heads accumulated per pass over the keys
template <typename T, int OB>
__global__ void __launch_bounds__(kValThreads, OB <= 2 ? 4 : (OB == 4 ? 3 : 2))
mix_values_kernel(const __grid_constant__ fr_mix_attn a, int row0, int max_keys, int n_blocks, int splits, int pass_keys,
                  const float* __restrict__ scores, const float2* __restrict__ stats, float* __restrict__ partial,
                  int32_t* __restrict__ counters) {
  extern __shared__ float sm[];
  const int rep = a.heads / a.kv_heads;
  const bool diff = a.mix == FR_MIX_DIFF;
  const int n_src = diff ? 2 * a.heads : a.heads;   // of the row
  const bool plain = a.mix == FR_MIX_PLAIN;
  const int my_src = diff ? 2 * rep : (plain ? rep : a.heads);  // that this kv head's outputs mix
  float* s_m = sm;                                  // [my_src]
  float* s_il = s_m + my_src;                       // [my_src]
  float* s_p = s_il + my_src;                       // [my_src][keys per pass]
  float* s_w = s_p + my_src * pass_keys;            // [OB][keys per pass]
  float* s_red = s_w + OB * pass_keys;              // [256][8], afterwards [vdim]
  int64_t* s_slot = reinterpret_cast<int64_t*>(s_red + kValThreads * 8 + 32);
  __shared__ float s_small[kValThreads / 32];
  __shared__ int s_last;
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int split = blockIdx.x, g = blockIdx.y, lrow = blockIdx.z, tid = threadIdx.x;
  const int64_t t = row0 + lrow;
  const int64_t i = a.pos[t];
  const Visible vis = visible_keys(a, i, max_keys);
  const int blocks = (vis.n + kKeyBlock - 1) / kKeyBlock;
  const int src0 = diff ? 2 * g * rep : (plain ? g * rep : 0);
  const int64_t srow = static_cast<int64_t>(lrow) * n_src + src0;
  for (int s = tid >> 5; s < my_src; s += kValThreads / 32) {
    const float2* st = stats + (srow + s) * n_blocks;
    float m = -INFINITY, l = 0.f;
    for (int b = tid & 31; b < blocks; b += 32) {
      const float2 v = st[b];
      const float mn = fmaxf(m, v.x);
      l = l * expf(m - mn) + v.y * expf(v.x - mn);  // the block maxima are finite
      m = mn;
    }
    const float mw = warp_max(m);
    l = warp_sum(m == -INFINITY ? 0.f : l * expf(m - mw));
    if ((tid & 31) == 0) {
      s_m[s] = mw;
      s_il[s] = 1.0f / l;
    }
  }
  const int b0 = static_cast<int>(static_cast<int64_t>(blocks) * split / splits);
  const int b1 = static_cast<int>(static_cast<int64_t>(blocks) * (split + 1) / splits);
  const int64_t table_row = a.req_rows[a.tok_req[t]];
  const int vgroups = a.vdim / 8;
  const int key_lanes = kValThreads / vgroups;
  const int vg = tid % vgroups, kl = tid / vgroups;
  const T* vc = static_cast<const T*>(a.v) + static_cast<int64_t>(g) * a.vdim + vg * 8;
  const int64_t part_row = (static_cast<int64_t>(lrow) * splits + split) * a.heads;
  for (int o0 = 0; o0 < rep; o0 += OB) {
    const int no = min(OB, rep - o0);
    float acc[OB][8] = {};
    for (int k0 = b0 * kKeyBlock; k0 < min(b1 * kKeyBlock, vis.n); k0 += pass_keys) {
      const int nk = min(pass_keys, min(b1 * kKeyBlock, vis.n) - k0);
      __syncthreads();
      for (int s = tid / 64; s < my_src; s += kValThreads / 64)
        for (int kk = tid % 64; kk < nk; kk += 64)
          s_p[s * pass_keys + kk] = expf(scores[(srow + s) * max_keys + k0 + kk] - s_m[s]) * s_il[s];
      if (tid < nk) s_slot[tid] = slot_of(a, table_row, vis.key(k0 + tid));
      __syncthreads();
      for (int o = tid / 64; o < no; o += kValThreads / 64)
        for (int kk = tid % 64; kk < nk; kk += 64) {
          float w = 0.f;
          if (diff) {
            w = s_p[2 * (o0 + o) * pass_keys + kk] - a.lambda * s_p[(2 * (o0 + o) + 1) * pass_keys + kk];
          } else if (plain) {
            w = s_p[(o0 + o) * pass_keys + kk];
          } else {
            const float* cf = a.coef + static_cast<int64_t>(g * rep + o0 + o) * a.heads;
            for (int s = 0; s < my_src; ++s) w = fmaf(__ldg(cf + s), s_p[s * pass_keys + kk], w);
          }
          s_w[o * pass_keys + kk] = w;
        }
      __syncthreads();
      if (kl < key_lanes) {
#pragma unroll 4
        for (int kk = kl; kk < nk; kk += key_lanes) {
          float v[8];
          load8<T>(vc + s_slot[kk] * a.ldv, v);
#pragma unroll
          for (int o = 0; o < OB; ++o)
            if (o < no) {
              const float w = s_w[o * pass_keys + kk];
#pragma unroll
              for (int x = 0; x < 8; ++x) acc[o][x] = fmaf(w, v[x], acc[o][x]);
            }
        }
      }
    }
#pragma unroll
    for (int o = 0; o < OB; ++o) {
      if (o >= no) break;
      const int head = g * rep + o0 + o;
      __syncthreads();
      if (kl < key_lanes) {
#pragma unroll
        for (int x = 0; x < 8; ++x) s_red[(kl * vgroups + vg) * 8 + x] = acc[o][x];
      }
      __syncthreads();
      float f[4];  // vdim <= 4 * 256
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = tid + n * kValThreads;
        f[n] = 0.f;
        if (c < a.vdim)
          for (int k = 0; k < key_lanes; ++k) f[n] += s_red[k * a.vdim + c];
      }
      if (splits > 1) {
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int c = tid + n * kValThreads;
          if (c < a.vdim) partial[(part_row + head) * a.vdim + c] = f[n];
        }
      } else {
        __syncthreads();
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int c = tid + n * kValThreads;
          if (c < a.vdim) s_red[c] = f[n];
        }
        __syncthreads();
        finish_head<T>(a, t, head, s_red, s_small);
      }
    }
  }
  if (splits <= 1) return;
  // the CTA that finishes last adds the shares, in order
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    int32_t* c = counters + static_cast<int64_t>(lrow) * a.kv_heads + g;
    s_last = atomicAdd(c, 1) == splits - 1;
    if (s_last) *c = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int o = 0; o < rep; ++o) {
    const int head = g * rep + o;
    __syncthreads();
    for (int c = tid; c < a.vdim; c += kValThreads) {
      float f = 0.f;
      for (int s = 0; s < splits; ++s)
        f += __ldcg(partial + ((static_cast<int64_t>(lrow) * splits + s) * a.heads + head) * a.vdim + c);
      s_red[c] = f;
    }
    __syncthreads();
    finish_head<T>(a, t, head, s_red, s_small);
  }
}

static int values_smem(const fr_mix_attn& a, int ob, int pass_keys) {
  const int rep = a.heads / a.kv_heads;
  const int my_src = a.mix == FR_MIX_DIFF ? 2 * rep : (a.mix == FR_MIX_PLAIN ? rep : a.heads);
  return (my_src * (2 + pass_keys) + ob * pass_keys + kValThreads * 8 + 32) * 4 + pass_keys * 8;
}

template <typename T, int OB>
static int launch_values(const fr_mix_attn& a, int row0, int n_rows, int max_keys, int n_blocks, int splits, const float* scores,
                         const float2* stats, float* partial, int32_t* counters, bool pdl, cudaStream_t stream) {
  int pass_keys = kValKeys;  // no more than a split has, and what leaves several CTAs per SM their shared memory
  const int share = ceil_div(n_blocks, splits) * kKeyBlock;
  while (pass_keys > kKeyBlock && (pass_keys / 2 >= share || values_smem(a, OB, pass_keys) > 56 * 1024)) pass_keys /= 2;
  const int smem = values_smem(a, OB, pass_keys);
  FR_CHECK_SUPPORTED(smem <= 200 * 1024);
  static PerDeviceFlag f;
  if (ensure_dyn_smem(f, mix_values_kernel<T, OB>, 200 * 1024) != FR_OK) return FR_ERR_CUDA;
  return launch_kernel(mix_values_kernel<T, OB>, dim3(splits, a.kv_heads, n_rows), kValThreads, smem, stream, pdl, a, row0, max_keys,
                       n_blocks, splits, pass_keys, scores, stats, partial, counters);
}

template <typename T>
static int launch_rows(const fr_mix_attn& a, int row0, int n_rows, int max_keys, int splits, float* scores, float2* stats,
                       float* partial, int32_t* counters, cudaStream_t stream) {
  const int rep = a.heads / a.kv_heads;
  const int n_blocks = ceil_div(max_keys, kKeyBlock);
  const int k_heads = a.mix == FR_MIX_DIFF ? 2 * a.kv_heads : a.kv_heads;
  const int64_t ctas = static_cast<int64_t>(n_blocks) * k_heads * n_rows;
  int per = ctas > device_sm_count() * 32 ? kMaxPer : 1;
  if (rep * (a.dim + per * kKeyBlock) * 4 > 40 * 1024) per = 1;
  const int s1 = rep * (a.dim + per * kKeyBlock) * 4;
  FR_CHECK_SUPPORTED(s1 <= 200 * 1024);
  static PerDeviceFlag f1;
  if (ensure_dyn_smem(f1, mix_scores_kernel<T>, 200 * 1024) != FR_OK) return FR_ERR_CUDA;
  const bool pdl = n_rows <= kPdlRows;
  if (launch_kernel(mix_scores_kernel<T>, dim3(ceil_div(n_blocks, per), k_heads, n_rows), 128, s1, stream, pdl, a, row0, max_keys,
                    n_blocks, per, scores, stats) != FR_OK)
    return FR_ERR_CUDA;
  if (rep == 1) return launch_values<T, 1>(a, row0, n_rows, max_keys, n_blocks, splits, scores, stats, partial, counters, pdl, stream);
  if (rep == 2) return launch_values<T, 2>(a, row0, n_rows, max_keys, n_blocks, splits, scores, stats, partial, counters, pdl, stream);
  if (rep <= 4) return launch_values<T, 4>(a, row0, n_rows, max_keys, n_blocks, splits, scores, stats, partial, counters, pdl, stream);
  return launch_values<T, 8>(a, row0, n_rows, max_keys, n_blocks, splits, scores, stats, partial, counters, pdl, stream);
}

// ---------------------------------------------------------------------------
// bf16 prompts on tcgen05. One CTA: up to 128 consecutive tokens of one request, one v head, the source maps its
// outputs mix one after the other. Roles as in attn_tc.cu: warp 0 = TMA producer, warp 1 = TMEM allocation and
// issue of S = Q K^T, warp 6 = issue of P V (one thread issuing both paced the tiles), warps 2..5 = one token per thread (TMEM lane == token). Per key tile of 64 (one cache page):
//     S = Q_s K_s^T (two TMEM buffers);  P = exp2(S - m) as bf16 over S;  O += P V, V as it lies in the cache
// (token rows, so the B operand is MN-major). After a map's last tile the threads take O / l and add
// coef[o, s] times it to the accumulators.
// ---------------------------------------------------------------------------
constexpr int kTcThreads = 224;
constexpr float kRescaleThreshold = 8.0f;
constexpr int kMaxOut = 8;
constexpr int kTcBarBytes = 288 + kPageList * 4;

struct TcPlan {
  int q_boxes, v_boxes;   // 64-column boxes of a q / k row and of a v row
  int q_bufs;             // Q tiles in shared memory: the next map's is loaded ahead, PLAIN has one map
  int v_cols;             // TMEM columns of O and of one accumulator
  int n_out;              // outputs per CTA (PLAIN: 1, which needs no accumulator)
  int out_blocks;         // CTAs along y per v head (TALK) or per head (DIFF)
  int staged;             // DIFF: the first map's result waits in shared memory (fp16), not in TMEM
  int stages;             // K and V stages
  int extra;              // bytes before Q that the staged rows need besides Q's first buffer (a multiple of 1024)
  int tmem_cols, smem;
};

static bool plan_tc(int mix, int heads, int kv_heads, int dim, int vdim, TcPlan* pl) {
  if (dim % 16 != 0 || vdim % 16 != 0 || dim <= 0 || vdim <= 0 || dim > 192 || vdim > 192) return false;
  const int rep = heads / kv_heads;
  pl->q_boxes = (dim + 63) / 64;
  pl->v_boxes = (vdim + 63) / 64;
  pl->v_cols = (vdim + 31) / 32 * 32;
  pl->staged = 0;
  pl->q_bufs = mix == FR_MIX_PLAIN ? 1 : 2;
  int fit = (512 - 2 * kTileN - pl->v_cols) / pl->v_cols;
  if (fit < 1) return false;
  if (fit > kMaxOut) fit = kMaxOut;
  const int outs = mix == FR_MIX_TALK ? rep : 1;
  const int blocks = (outs + fit - 1) / fit;
  pl->n_out = (outs + blocks - 1) / blocks;
  pl->out_blocks = blocks;
  int need = 2 * kTileN + pl->v_cols * (mix == FR_MIX_PLAIN ? 1 : 1 + pl->n_out);
  if (mix == FR_MIX_DIFF && need > 256 && need - pl->v_cols <= 256) {  // without the accumulator two CTAs share an SM
    pl->staged = 1;
    need -= pl->v_cols;
  }
  pl->tmem_cols = need <= 256 ? 256 : 512;
  for (pl->stages = 4;; --pl->stages) {
    pl->smem = 1024 + pl->q_bufs * pl->q_boxes * kM * 128 + pl->stages * (pl->q_boxes + pl->v_boxes) * kTileN * 128 + kTcBarBytes;
    pl->extra = pl->staged && kM * pl->v_cols * 2 > pl->q_boxes * kM * 128 ? kM * pl->v_cols * 2 - pl->q_boxes * kM * 128 : 0;
    pl->smem += pl->extra;
    if (pl->stages == 2 || pl->smem <= (pl->tmem_cols == 256 ? 112 : 227) * 1024) break;
  }
  if (pl->tmem_cols == 512 && pl->smem < 116 * 1024) pl->smem = 116 * 1024;  // one CTA per SM owns all of TMEM
  return pl->smem <= 227 * 1024;
}

template <bool BIAS>
__global__ void __launch_bounds__(kTcThreads, 2)
mix_tc_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
              const __grid_constant__ CUtensorMap tv, const __grid_constant__ fr_mix_attn a, const TcPlan pl,
              const int32_t* __restrict__ tiles, int* status) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = ptx::smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const int q_bytes = pl.q_boxes * kM * 128, k_bytes = pl.q_boxes * kTileN * 128, v_bytes = pl.v_boxes * kTileN * 128;
  const int n_st = pl.stages;
  const uint32_t sm_q = base + pl.extra, sm_k = sm_q + pl.q_bufs * q_bytes, sm_v = sm_k + n_st * k_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + pl.extra + pl.q_bufs * q_bytes + n_st * (k_bytes + v_bytes));
  const uint32_t bar0 = ptx::smem_u32(bars);
  const uint32_t bar_qfull = bar0, bar_qempty = bar0 + 16;    // [2] each
  const uint32_t bar_sfull = bar0 + 32;                       // [2]
  const uint32_t bar_kfull = bar0 + 48, bar_kempty = bar0 + 80;   // [stages <= 4] each
  const uint32_t bar_vfull = bar0 + 112, bar_vempty = bar0 + 144;
  const uint32_t bar_ofull = bar0 + 176;                      // [2] P.V accumulated, by S buffer
  // P written (128 arrivals), one per S buffer: the softmax threads may finish two tiles while the issuing thread
  // still waits for V, and a single barrier would then be two phases ahead of its parity wait
  const uint32_t bar_pfull = bar0 + 192;                      // [2]
  const uint32_t bar_oread = bar0 + 208;                      // O read out (128 arrivals), one phase per map
  const uint32_t bar_done = bar0 + 216;                       // a map's last P.V, one phase per map
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 32);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* pages = reinterpret_cast<int*>(bars + 36);
  // staged: [128 rows][v_cols] fp16, 16-byte chunks swizzled by row, in `extra` bytes and Q's first buffer behind them,
  // which the first map is done with
  uint8_t* stage_rows = smem;
  ptx::griddep_wait();
  ptx::griddep_launch_dependents();
  const int rep = a.heads / a.kv_heads;
  const bool diff = a.mix == FR_MIX_DIFF, plain = a.mix == FR_MIX_PLAIN;
  // x: tile, y: DIFF head; TALK (v head, block of its outputs). PLAIN: the heads of a tile side by side, the last
  // tiles (with the most keys below the causal edge) first
  int tile = blockIdx.x, by = blockIdx.y;
  if (plain) {
    const int id = static_cast<int>(blockIdx.y * gridDim.x + blockIdx.x);
    tile = static_cast<int>(gridDim.x) - 1 - id / a.heads;
    by = id % a.heads;
  }
  const int vh = diff || plain ? by / rep : by / pl.out_blocks;
  const int out0 = diff || plain ? by : vh * rep + by % pl.out_blocks * pl.n_out;
  const int n_out = diff || plain ? 1 : min(pl.n_out, (vh + 1) * rep - out0);
  const int n_src = diff ? 2 : (plain ? 1 : a.heads);
  const int src0 = diff ? 2 * out0 : (plain ? out0 : 0);
  const int req = tiles[3 * tile], row0 = tiles[3 * tile + 1], n_tok = tiles[3 * tile + 2];
  const int pos0 = static_cast<int>(a.pos[row0]);
  const int pos_last = pos0 + n_tok - 1;
  const int32_t* table = a.req_to_token + a.req_rows[req] * a.table_stride;
  const KeyTiles kt = key_tiles(a, pos0, pos_last);  // every role derives the same list
  const int n_tiles = kt.n;
  const int total = n_tiles * n_src;
  auto k_head = [&](int s) { return diff ? 2 * vh + s : (plain ? vh : s / rep); };

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 24; ++i) ptx::mbar_init(bar0 + 8 * i, 1);
    ptx::mbar_init(bar_pfull, 128);
    ptx::mbar_init(bar_pfull + 8, 128);
    ptx::mbar_init(bar_oread, 128);
    ptx::mbar_init(bar_done, 1);
    *abort_flag = 0;
    ptx::mbar_init_fence();
    ptx::prefetch_tmap(&tq);
    ptx::prefetch_tmap(&tk);
    ptx::prefetch_tmap(&tv);
  }
  load_pages(a, table, kt, pages);
  if (warp == 1) {
    __syncwarp();
    ptx::tmem_alloc(ptx::smem_u32(tmem_slot), pl.tmem_cols);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t col_o = tmem_base + 2 * kTileN;
  const uint32_t col_acc = col_o + pl.v_cols;

  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      auto load_q = [&](int s) -> bool {
        const uint32_t st = s & 1;
        if (!ptx::mbar_wait(bar_qempty + 8 * st, ((s >> 1) & 1) ^ 1u, abort_flag, status, 71)) return false;
        ptx::mbar_expect_tx(bar_qfull + 8 * st, q_bytes);
        for (int b = 0; b < pl.q_boxes; ++b)
          ptx::tma_load_2d(sm_q + st * q_bytes + b * kM * 128, &tq, (src0 + s) * a.dim + b * 64, row0, bar_qfull + 8 * st);
        return true;
      };
      // stage and parity of the next K and V tile, position of the next K tile (map, tile): counted, not divided
      int k_st = 0, k_ph = 0, k_j = 0, k_s = 0, next_k = 0;
      auto load_k = [&]() -> bool {
        if (k_j == 0 && !load_q(k_s)) return false;
        if (!ptx::mbar_wait(bar_kempty + 8 * k_st, k_ph ^ 1u, abort_flag, status, 72)) return false;
        ptx::mbar_expect_tx(bar_kfull + 8 * k_st, k_bytes);
        const int row = page_at(a, table, kt, pages, k_j), col = k_head(k_s) * a.dim;
        for (int b = 0; b < pl.q_boxes; ++b)
          ptx::tma_load_2d(sm_k + k_st * k_bytes + b * kTileN * 128, &tk, col + b * 64, row, bar_kfull + 8 * k_st);
        if (++k_st == n_st) { k_st = 0; k_ph ^= 1; }
        if (++k_j == n_tiles) { k_j = 0; ++k_s; }
        ++next_k;
        return true;
      };
      // K (and at a map's start its Q) runs up to n_st - 1 tiles ahead of V
      int v_st = 0, v_ph = 0, v_j = 0;
      for (int it = 0; it < total && ok; ++it) {
        while (ok && next_k < total && next_k < it + n_st) ok = load_k();
        if (!ok) break;
        ok = ptx::mbar_wait(bar_vempty + 8 * v_st, v_ph ^ 1u, abort_flag, status, 73);
        if (!ok) break;
        ptx::mbar_expect_tx(bar_vfull + 8 * v_st, v_bytes);
        const int row = page_at(a, table, kt, pages, v_j);
        for (int b = 0; b < pl.v_boxes; ++b)
          ptx::tma_load_2d(sm_v + v_st * v_bytes + b * kTileN * 128, &tv, vh * a.vdim + b * 64, row, bar_vfull + 8 * v_st);
        if (++v_st == n_st) { v_st = 0; v_ph ^= 1; }
        if (++v_j == n_tiles) v_j = 0;
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = ptx::make_idesc(1u, 1u, kM, kTileN);
      const int k_steps = a.dim / 16;
      bool ok = true;
      int st = 0, ph = 0, j = 0, s = 0;
      for (int it = 0; it < total && ok; ++it) {
        const uint32_t sb = it & 1;
        if (j == 0) ok = ptx::mbar_wait(bar_qfull + 8 * (s & 1), (s >> 1) & 1, abort_flag, status, 74);
        ok = ok && ptx::mbar_wait(bar_kfull + 8 * st, ph, abort_flag, status, 75);
        // the buffer held P of tile it - 2
        if (ok && it >= 2) ok = ptx::mbar_wait(bar_ofull + 8 * sb, ((it >> 1) - 1) & 1, abort_flag, status, 83);
        if (!ok) break;
        ptx::tc_fence_after();
        const uint64_t a_desc = ptx::smem_desc_sw128(sm_q + (s & 1) * q_bytes);
        const uint64_t b_desc = ptx::smem_desc_sw128(sm_k + st * k_bytes);
        const uint32_t d = tmem_base + sb * kTileN;
#pragma unroll 1
        for (int kb = 0; kb < k_steps; kb += 4) {  // 64 columns per box; descriptor addresses count 16-byte units
          const uint64_t ad = a_desc + (kb >> 2) * (kM * 128 / 16), bd = b_desc + (kb >> 2) * (kTileN * 128 / 16);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (kb + k < k_steps) ptx::mma_f16(d, ad + 2u * k, bd + 2u * k, idesc_s, (kb | k) != 0 ? 1u : 0u);
        }
        ptx::tc_commit(bar_sfull + 8 * sb);
        ptx::tc_commit(bar_kempty + 8 * st);
        if (++st == n_st) { st = 0; ph ^= 1; }
        if (++j == n_tiles) {
          ptx::tc_commit(bar_qempty + 8 * (s & 1));
          j = 0;
          ++s;
        }
      }
    }
    __syncwarp();
  } else if (warp == 6) {
    if (lane == 0) {
      const uint32_t idesc_o = ptx::make_idesc(1u, 1u, kM, a.vdim) | (1u << 16);  // B is MN-major
      bool ok = true;
      int st = 0, ph = 0, j = 0, s = 0;
      for (int it = 0; it < total && ok; ++it) {
        const uint32_t sb = it & 1;
        ok = ptx::mbar_wait(bar_vfull + 8 * st, ph, abort_flag, status, 77) &&
             ptx::mbar_wait(bar_pfull + 8 * sb, (it >> 1) & 1, abort_flag, status, 76);
        // the first P.V of a map overwrites O: the previous map's must have been read
        if (ok && j == 0 && s > 0) ok = ptx::mbar_wait(bar_oread, (s - 1) & 1, abort_flag, status, 78);
        if (!ok) break;
        ptx::tc_fence_after();
        const uint64_t v_desc = smem_desc_mn(sm_v + st * v_bytes, kTileN * 128);
#pragma unroll
        for (int k = 0; k < kTileN / 16; ++k)  // 16 keys = 8 columns of P, 16 rows of V
          ptx::mma_f16_ts(col_o, tmem_base + sb * kTileN + 8u * k, v_desc + static_cast<uint64_t>(k * 16 * 128 >> 4), idesc_o,
                          (j | k) != 0 ? 1u : 0u);
        ptx::tc_commit(bar_ofull + 8 * sb);
        ptx::tc_commit(bar_vempty + 8 * st);
        if (++st == n_st) { st = 0; ph ^= 1; }
        if (++j == n_tiles) {
          ptx::tc_commit(bar_done);
          j = 0;
          ++s;
        }
      }
    }
    __syncwarp();
  } else {
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const bool live = r < n_tok;
    const int i = pos0 + min(r, n_tok - 1);
    const int lo = static_cast<int>(lowest_key(a, i));
    const int keep = a.mask == FR_MASK_CHUNK ? 0 : a.keep_first;
    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    const float scale = a.scale * kLog2e;
    auto wait_all = [&](uint32_t bar, uint32_t parity, int site) -> bool {
      int okw = 0;
      if (lane == 0) okw = ptx::mbar_wait(bar, parity, abort_flag, status, site) ? 1 : 0;
      okw = __shfl_sync(0xffffffffu, okw, 0);
      ptx::tc_fence_after();
      return okw != 0;
    };
    bool ok = true;
    const int chunk_mask = pl.v_cols % 64 == 0 ? 7 : 3;  // swizzle within 128 (or 64) bytes of a row
    __nv_bfloat16* out_row = static_cast<__nv_bfloat16*>(a.out) + (row0 + min(r, n_tok - 1)) * a.ldo +
                             static_cast<int64_t>(out0) * a.vdim;
    for (int s = 0; s < n_src && ok; ++s) {
      float m_used = -INFINITY, l_sum = 0.f;
      const float slope = BIAS && a.slopes != nullptr ? a.slopes[src0 + s] * kLog2e : 0.f;
      for (int j = 0; j < n_tiles; ++j) {
        const int it = s * n_tiles + j;
        const uint32_t st = it & 1;
        ok = wait_all(bar_sfull + 8 * st, (it >> 1) & 1, 79);
        if (!ok) break;
        uint32_t s0[32], s1[32];
        ptx::tmem_ld_32x32(tmem_base + lane_off + st * kTileN, s0);
        ptx::tmem_ld_32x32(tmem_base + lane_off + st * kTileN + 32, s1);
        ptx::tmem_ld_wait();
        const int j0 = kt.at(j) * kTileN;
        const float bias0 = slope * static_cast<float>(j0 - i);
        auto sv = [&](int c) -> uint32_t& { return c < 32 ? s0[c & 31] : s1[c & 31]; };
        if constexpr (BIAS) {
#pragma unroll
          for (int c = 0; c < 64; ++c)
            sv(c) = __float_as_uint(fmaf(__uint_as_float(sv(c)), scale, fmaf(slope, static_cast<float>(c), bias0)));
        }
        const bool partly = j0 + kTileN - 1 > i || (j0 < lo && j0 + kTileN > keep);
        if (__any_sync(0xffffffffu, partly)) {
          const uint64_t vis = visible_bits(j0, i, lo, keep);
          const uint32_t v0 = static_cast<uint32_t>(vis), v1 = static_cast<uint32_t>(vis >> 32);
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            if (!((v0 >> c) & 1u)) s0[c] = 0xff800000u;  // -inf
            if (!((v1 >> c) & 1u)) s1[c] = 0xff800000u;
          }
        }
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int c = 0; c < 32; ++c) mx[c & 3] = max3(mx[c & 3], __uint_as_float(s0[c]), __uint_as_float(s1[c]));
        const float mraw = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
        const float tmax = BIAS ? mraw : mraw * scale;  // without bias the scale (> 0) is applied with the maximum
        float factor = 1.0f;
        if (tmax > m_used + kRescaleThreshold) {  // false while nothing is visible (both -inf)
          factor = ex2(m_used - tmax);            // 0 at the first visible tile
          m_used = tmax;
        }
        l_sum *= factor;
        if (j > 0 && __any_sync(0xffffffffu, factor != 1.0f)) {
          ok = wait_all(bar_ofull + 8 * (st ^ 1u), ((it - 1) >> 1) & 1, 80);
          if (!ok) break;
#pragma unroll 1
          for (int c = 0; c < pl.v_cols / 32; ++c) {
            uint32_t o[32];
            ptx::tmem_ld_32x32(col_o + lane_off + c * 32, o);
            ptx::tmem_ld_wait();
#pragma unroll
            for (int x = 0; x < 32; ++x) o[x] = __float_as_uint(__uint_as_float(o[x]) * factor);
            ptx::tmem_st_32x32(col_o + lane_off + c * 32, o);
          }
          ptx::tmem_st_wait();
        }
        const float m_ref = m_used == -INFINITY ? 0.f : m_used;  // nothing visible yet: every weight is 2^-inf = 0
        uint64_t ps[4] = {0ull, 0ull, 0ull, 0ull};
        const uint64_t scale2 = pack_f32x2(scale, scale), neg_m2 = pack_f32x2(-m_ref, -m_ref);
        uint32_t w[32];
#pragma unroll
        for (int x = 0; x < 32; ++x) {
          const uint64_t z = pack_f32x2(__uint_as_float(sv(2 * x)), __uint_as_float(sv(2 * x + 1)));
          float p0, p1;
          unpack_f32x2(BIAS ? add_f32x2(z, neg_m2) : fma_f32x2(z, scale2, neg_m2), p0, p1);
          p0 = ex2(p0);
          p1 = ex2(p1);
          ps[x & 3] = add_f32x2(ps[x & 3], pack_f32x2(p0, p1));
          w[x] = pack_bf16(p0, p1);
        }
        float ps0, ps1;
        unpack_f32x2(add_f32x2(add_f32x2(ps[0], ps[1]), add_f32x2(ps[2], ps[3])), ps0, ps1);
        l_sum += ps0 + ps1;
        ptx::tmem_st_32x32(tmem_base + lane_off + st * kTileN, w);
        ptx::tmem_st_wait();
        ptx::tc_fence_before();
        ptx::mbar_arrive(bar_pfull + 8 * st);
      }
      if (!ok) break;
      ok = wait_all(bar_done, s & 1, 81);
      if (!ok) break;
      const float inv = 1.0f / l_sum;
      if (plain) {
        const float scl = inv * head_gate_of(a, row0 + min(r, n_tok - 1), out0);
#pragma unroll 1
        for (int c = 0; c < pl.v_cols / 32; ++c) {
          uint32_t o[32];
          ptx::tmem_ld_32x32(col_o + lane_off + c * 32, o);
          ptx::tmem_ld_wait();
#pragma unroll
          for (int x = 0; x < 2; ++x) {  // 16 columns: one 32-byte store
            uint32_t w8[8];
#pragma unroll
            for (int e = 0; e < 8; ++e)
              w8[e] = pack_bf16(__uint_as_float(o[16 * x + 2 * e]) * scl, __uint_as_float(o[16 * x + 2 * e + 1]) * scl);
            if (live && c * 32 + x * 16 < a.vdim) ptx::st_global_v8(out_row + c * 32 + x * 16, w8);
          }
          __syncwarp();
        }
        ptx::tc_fence_before();
        continue;
      }
      if (pl.staged) {
        // first map: a1 as fp16 into this thread's own row of shared memory; second map: a1 - lambda a2, scaled by its
        // root mean square, into the output (two passes over O)
        uint8_t* row = stage_rows + r * pl.v_cols * 2;
        auto chunk = [&](int c) { return reinterpret_cast<uint4*>(row + (((c & ~chunk_mask) | ((c ^ r) & chunk_mask)) << 4)); };
        float ss = 0.f;
        for (int pass = s == 0 ? 1 : 0; pass < 2; ++pass) {
          const float scl = s == 0 ? inv : a.out_scale / sqrtf(ss / static_cast<float>(a.vdim_true) + a.eps);
#pragma unroll 1
          for (int c = 0; c < pl.v_cols / 32; ++c) {
            uint32_t o[32];
            ptx::tmem_ld_32x32(col_o + lane_off + c * 32, o);
            ptx::tmem_ld_wait();
            if (s == 0) {
#pragma unroll
              for (int x = 0; x < 4; ++x) {
                uint32_t w4[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  const __half2 h = __floats2half2_rn(__uint_as_float(o[8 * x + 2 * e]) * scl,
                                                      __uint_as_float(o[8 * x + 2 * e + 1]) * scl);
                  w4[e] = *reinterpret_cast<const uint32_t*>(&h);
                }
                *chunk(c * 4 + x) = make_uint4(w4[0], w4[1], w4[2], w4[3]);
              }
            } else {
#pragma unroll
              for (int x = 0; x < 2; ++x) {  // 16 columns: one 32-byte store
                uint32_t w8[8];
                const bool valid = c * 32 + x * 16 < a.vdim;
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                  const uint4 first = *chunk(c * 4 + 2 * x + y);
                  const uint32_t fw[4] = {first.x, first.y, first.z, first.w};
#pragma unroll
                  for (int e = 0; e < 4; ++e) {
                    const int q = 16 * x + 8 * y + 2 * e;
                    const float2 a1 = __half22float2(*reinterpret_cast<const __half2*>(&fw[e]));
                    const float f0 = fmaf(-a.lambda * inv, __uint_as_float(o[q]), a1.x);
                    const float f1 = fmaf(-a.lambda * inv, __uint_as_float(o[q + 1]), a1.y);
                    if (valid) ss = pass == 0 ? fmaf(f0, f0, fmaf(f1, f1, ss)) : ss;
                    w8[4 * y + e] = pack_bf16(f0 * scl, f1 * scl);
                  }
                }
                if (live && valid && pass == 1) ptx::st_global_v8(out_row + c * 32 + x * 16, w8);
              }
            }
            __syncwarp();
          }
        }
        ptx::tc_fence_before();
        ptx::mbar_arrive(bar_oread);
        continue;
      }
#pragma unroll 1
      for (int c = 0; c < pl.v_cols / 32; ++c) {
        uint32_t o[32];
        ptx::tmem_ld_32x32(col_o + lane_off + c * 32, o);
        ptx::tmem_ld_wait();
#pragma unroll 1
        for (int n = 0; n < n_out; ++n) {
          const float cf = inv * (diff ? (s == 0 ? 1.0f : -a.lambda)
                                       : __ldg(a.coef + static_cast<int64_t>(out0 + n) * a.heads + s));
          uint32_t acc[32];
          if (s > 0) {
            ptx::tmem_ld_32x32(col_acc + lane_off + n * pl.v_cols + c * 32, acc);
            ptx::tmem_ld_wait();
          } else {
#pragma unroll
            for (int x = 0; x < 32; ++x) acc[x] = 0u;
          }
#pragma unroll
          for (int x = 0; x < 32; ++x)
            acc[x] = __float_as_uint(fmaf(cf, __uint_as_float(o[x]), __uint_as_float(acc[x])));
          ptx::tmem_st_32x32(col_acc + lane_off + n * pl.v_cols + c * 32, acc);
        }
        ptx::tmem_st_wait();
      }
      ptx::tc_fence_before();
      ptx::mbar_arrive(bar_oread);
    }
    if (ok && !pl.staged && !plain) {
      for (int n = 0; n < n_out; ++n) {
        float scl = 1.0f;
        if (diff) {
          float ss = 0.f;
#pragma unroll 1
          for (int c = 0; c < pl.v_cols / 32; ++c) {
            uint32_t o[32];
            ptx::tmem_ld_32x32(col_acc + lane_off + n * pl.v_cols + c * 32, o);
            ptx::tmem_ld_wait();
#pragma unroll
            for (int x = 0; x < 32; ++x)
              if (c * 32 + x < a.vdim) ss = fmaf(__uint_as_float(o[x]), __uint_as_float(o[x]), ss);
          }
          scl = a.out_scale / sqrtf(ss / static_cast<float>(a.vdim_true) + a.eps);
        }
        __nv_bfloat16* dst = out_row + static_cast<int64_t>(n) * a.vdim;
#pragma unroll 1
        for (int c = 0; c < pl.v_cols / 32; ++c) {
          uint32_t o[32];
          ptx::tmem_ld_32x32(col_acc + lane_off + n * pl.v_cols + c * 32, o);
          ptx::tmem_ld_wait();
          if (live) {
            uint4* d4 = reinterpret_cast<uint4*>(dst + c * 32);
#pragma unroll
            for (int x = 0; x < 4; ++x)
              if (c * 32 + x * 8 < a.vdim)
                d4[x] = make_uint4(pack_bf16(__uint_as_float(o[8 * x]) * scl, __uint_as_float(o[8 * x + 1]) * scl),
                                   pack_bf16(__uint_as_float(o[8 * x + 2]) * scl, __uint_as_float(o[8 * x + 3]) * scl),
                                   pack_bf16(__uint_as_float(o[8 * x + 4]) * scl, __uint_as_float(o[8 * x + 5]) * scl),
                                   pack_bf16(__uint_as_float(o[8 * x + 6]) * scl, __uint_as_float(o[8 * x + 7]) * scl));
          }
          __syncwarp();
        }
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
    ptx::tmem_dealloc(tmem_base, pl.tmem_cols);
  }
}

static int check_args(const fr_mix_attn* a) {
  FR_CHECK_ARG(a && (a->dtype == 0 || a->dtype == 1) && a->mix >= FR_MIX_DIFF && a->mix <= FR_MIX_PLAIN);
  FR_CHECK_ARG((a->mask == FR_MASK_WINDOW || a->mask == FR_MASK_CHUNK) && a->mask_size > 0 && a->keep_first >= 0);
  FR_CHECK_ARG(a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0);
  FR_CHECK_ARG(a->dim > 0 && a->dim % 16 == 0 && a->vdim > 0 && a->vdim % 16 == 0 && a->vdim_true > 0);
  FR_CHECK_ARG(a->q && a->k && a->v && a->out && a->req_to_token && a->req_rows && a->tok_req && a->pos && a->num_slots > 0);
  FR_CHECK_ARG(aligned16(a->q) && aligned16(a->k) && aligned16(a->v) && aligned16(a->out) && a->ldq % 8 == 0 &&
               a->ldk % 8 == 0 && a->ldv % 8 == 0 && a->ldo % 8 == 0);
  FR_CHECK_ARG(a->mix != FR_MIX_TALK || a->coef);
  FR_CHECK_ARG(a->head_gate == nullptr || (a->mix == FR_MIX_PLAIN && a->ld_gate >= a->heads));
  return FR_OK;
}

}  // namespace mix
}  // namespace fr

using namespace fr;

extern "C" int64_t fr_mix_attn_rows_scratch(int mix_kind, int heads, int vdim, int n_rows, int max_keys, int splits) {
  if (heads <= 0 || vdim <= 0 || n_rows < 0 || max_keys <= 0 || splits <= 0) return -1;
  const int64_t src = static_cast<int64_t>(n_rows) * (mix_kind == FR_MIX_DIFF ? 2 * heads : heads);
  const int64_t stats = src * ceil_div(max_keys, mix::kKeyBlock) * 8;
  const int64_t part = splits > 1 ? static_cast<int64_t>(n_rows) * splits * heads * vdim * 4 : 0;
  return stats + src * max_keys * 4 + part;
}

extern "C" int fr_mix_attn_rows(const fr_mix_attn* a, int row0, int n_rows, int max_keys, int splits, void* scratch,
                                int64_t scratch_bytes, int32_t* counters, cudaStream_t stream) {
  const int st = mix::check_args(a);
  if (st != FR_OK) return st;
  FR_CHECK_ARG(row0 >= 0 && n_rows >= 0 && max_keys > 0 && splits > 0);
  if (n_rows == 0) return FR_OK;
  FR_CHECK_ARG(scratch && aligned16(scratch) && (splits == 1 || counters));
  FR_CHECK_ARG(scratch_bytes >= fr_mix_attn_rows_scratch(a->mix, a->heads, a->vdim, n_rows, max_keys, splits));
  FR_CHECK_SUPPORTED(a->vdim <= 1024 && n_rows <= 65535);
  const int64_t src = static_cast<int64_t>(n_rows) * (a->mix == FR_MIX_DIFF ? 2 * a->heads : a->heads);
  float2* stats = static_cast<float2*>(scratch);
  float* scores = reinterpret_cast<float*>(stats + src * ceil_div(max_keys, mix::kKeyBlock));
  float* partial = scores + src * max_keys;
  return a->dtype == 0 ? mix::launch_rows<__nv_bfloat16>(*a, row0, n_rows, max_keys, splits, scores, stats, partial, counters, stream)
                       : mix::launch_rows<float>(*a, row0, n_rows, max_keys, splits, scores, stats, partial, counters, stream);
}

extern "C" int fr_mix_attn_tc_fits(int mix_kind, int heads, int kv_heads, int dim, int vdim) {
  mix::TcPlan pl;
  return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && mix::plan_tc(mix_kind, heads, kv_heads, dim, vdim, &pl) ? 1 : 0;
}

extern "C" int64_t fr_mix_attn_tc_scratch(const fr_mix_attn* a, int n_tiles, int max_pos, int64_t budget) {
  if (a == nullptr || a->heads <= 0 || a->kv_heads <= 0 || a->mask_size <= 0 || n_tiles <= 0 || max_pos < 0) return 0;
  mix::TcPlan pl;
  if (a->mix != FR_MIX_TALK || !mix::plan_tc(a->mix, a->heads, a->kv_heads, a->dim, a->vdim, &pl)) return 0;
  if (a->kv_heads * pl.out_blocks < 2) return 0;  // every map is computed once as it is
  const int64_t per_tile = talk_tc_tile_bytes(*a, max_pos);
  int64_t tiles = budget / per_tile;
  if (tiles > n_tiles) tiles = n_tiles;
  // too few tiles at a time leave SMs idle: the maps are recomputed per v head instead
  return tiles < n_tiles && tiles * a->heads < 96 ? 0 : tiles * per_tile;
}

extern "C" int fr_mix_attn_tc(const fr_mix_attn* a, const int32_t* tiles, int n_tiles, int n_rows, int max_pos, void* scratch,
                              int64_t scratch_bytes, cudaStream_t stream) {
  const int st = mix::check_args(a);
  if (st != FR_OK) return st;
  FR_CHECK_ARG(tiles && n_tiles >= 0 && n_rows >= 0);
  FR_CHECK_ARG((reinterpret_cast<uintptr_t>(a->out) & 31u) == 0 && a->ldo % 16 == 0);  // 32-byte stores
  if (n_tiles == 0 || n_rows == 0) return FR_OK;
  mix::TcPlan pl;
  FR_CHECK_SUPPORTED(a->dtype == 0 && a->num_slots >= mix::kTileN &&
                     mix::plan_tc(a->mix, a->heads, a->kv_heads, a->dim, a->vdim, &pl));
  if (scratch != nullptr && scratch_bytes > 0) {
    FR_CHECK_ARG(a->mix == FR_MIX_TALK && aligned16(scratch) && max_pos >= 0);
    return talk_tc(*a, tiles, n_tiles, n_rows, max_pos, scratch, scratch_bytes, stream);
  }
  const bool diff = a->mix == FR_MIX_DIFF;
  const int n_src = diff ? 2 * a->heads : a->heads, k_heads = diff ? 2 * a->kv_heads : a->kv_heads;
  CUtensorMap tq, tk, tv;
  int r = make_tmap_bf16_box64(&tq, a->q, static_cast<uint64_t>(n_src) * a->dim, n_rows, a->ldq, mix::kM);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tk, a->k, static_cast<uint64_t>(k_heads) * a->dim, a->num_slots, a->ldk, mix::kTileN);
  if (r == FR_OK) r = make_tmap_bf16_box64(&tv, a->v, static_cast<uint64_t>(a->kv_heads) * a->vdim, a->num_slots, a->ldv, mix::kTileN);
  if (r != FR_OK) return r;
  int* status = device_status_ptr();
  if (!status) return FR_ERR_CUDA;
  dim3 grid(n_tiles, a->mix == FR_MIX_TALK ? a->kv_heads * pl.out_blocks : a->heads);
  static PerDeviceFlag f0, f1;
  if (a->slopes != nullptr || !(a->scale > 0.f)) {
    if (ensure_dyn_smem(f1, mix::mix_tc_kernel<true>, 227 * 1024) != FR_OK) return FR_ERR_CUDA;
    return launch_kernel(mix::mix_tc_kernel<true>, grid, mix::kTcThreads, pl.smem, stream, n_rows <= kPdlRows, tq, tk, tv, *a, pl,
                         tiles, status);
  } else {
    if (ensure_dyn_smem(f0, mix::mix_tc_kernel<false>, 227 * 1024) != FR_OK) return FR_ERR_CUDA;
    return launch_kernel(mix::mix_tc_kernel<false>, grid, mix::kTcThreads, pl.smem, stream, n_rows <= kPdlRows, tq, tk, tv, *a, pl,
                         tiles, status);
  }
}
