// Latent attention: one cached row per token, [latent (rank) | rotated key (rot)], shared by
// all heads.  With the key and value projections of a head taken into its query and its
// output ("absorbed"), a head's query is [W_uk^T q | rotated q], its keys are the cached rows
// and its values the first `rank` channels of them.
//
//   latent_prepare_kernel   norm of the latent, rotation of the shared key, store; rotation
//                           (and copy) of the queries; _vec: the same 16 bytes at a time
//   latent_gather_kernel    cached rows of a batch's sequences side by side
//   latent_attn_kernel      absorbed attention, bf16: portions and single tokens alike.  A
//                           CTA owns 16 (token, head) rows of one sequence and a range of
//                           keys; tiles of cached rows come through a ring and serve as K
//                           and as V.  Waits are bounded
//   latent_merge_kernel     key ranges of a row -> one result
//
// Scores, softmax weights and sums are fp32; the weights enter the tensor product with the
// values as two bf16 parts.
#include "fk_types.cuh"

#include <cmath>
#include <mutex>
#include <vector>

namespace fk {

struct LatentPrepParams {
  const void* q; const void* lat; int64_t in_stride;  // packed projection rows
  int q_pitch;                                        // elements between heads of q
  const float* weight;                                // [rank]
  const float* cos_sin; int64_t max_position;         // [max_position, rot] = cos | sin
  const int32_t* slots; const int64_t* positions;
  void* cache; int64_t num_slots; int cache_pitch;
  void* q_out; int q_out_pitch, q_rot_at, copy;       // copy: unrotated channels to column 0
  int64_t rows; int heads, dim, rot, rank;
  float eps;
  int32_t* status;
};

// One warp per (token, head), and one more per token for the cached row.
template <typename T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const LatentPrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (h > p.heads) return;
  const int half = p.rot >> 1;
  for (int64_t t = blockIdx.y; t < p.rows; t += gridDim.y) {
    int64_t pos = p.positions[t];
    if (pos < 0 || pos >= p.max_position) {
      if (lane == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_POSITION);
      pos = 0;
    }
    const float* cs = p.cos_sin + pos * p.rot;
    const T* src;
    T* dst;
    if (h < p.heads) {
      const T* q = static_cast<const T*>(p.q) + t * p.in_stride + (int64_t)h * p.q_pitch;
      T* out = static_cast<T*>(p.q_out) + (t * p.heads + h) * p.q_out_pitch;
      if (p.copy)
        for (int c = lane; c < p.dim; c += 32) out[c] = q[c];
      for (int c = p.q_rot_at + p.rot + lane; c < p.q_out_pitch; c += 32)
        Elem<T>::store(out + c, 0.f);
      src = q + p.dim;
      dst = out + p.q_rot_at;
    } else {
      const int64_t slot = p.slots[t];
      if (slot < 0 || slot >= p.num_slots) {
        if (slot >= p.num_slots && lane == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
        continue;
      }
      const T* c0 = static_cast<const T*>(p.lat) + t * p.in_stride;
      T* out = static_cast<T*>(p.cache) + slot * p.cache_pitch;
      float ss = 0.f;
      for (int c = lane; c < p.rank; c += 32) {
        const float x = Elem<T>::load(c0 + c);
        ss += x * x;
      }
      const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)p.rank + p.eps);
      for (int c = lane; c < p.rank; c += 32)
        Elem<T>::store(out + c, Elem<T>::load(c0 + c) * rs * p.weight[c]);
      for (int c = p.rank + p.rot + lane; c < p.cache_pitch; c += 32)
        Elem<T>::store(out + c, 0.f);
      src = c0 + p.rank;
      dst = out + p.rank;
    }
    for (int i = lane; i < half; i += 32) {
      const float u = Elem<T>::load(src + 2 * i), v = Elem<T>::load(src + 2 * i + 1);
      const float c = cs[i], s = cs[half + i];
      Elem<T>::store(dst + 2 * i, u * c - v * s);
      Elem<T>::store(dst + 2 * i + 1, v * c + u * s);
    }
  }
}

// All sizes multiples of 8, bf16: 16 bytes a thread.  blockIdx.x 0: the queries of a token;
// 1: the cached rows of 8 tokens, a warp each.
__global__ void __launch_bounds__(256) latent_prepare_vec_kernel(const LatentPrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = p.rot >> 1;
  auto rotated = [&](const uint16_t* src, int64_t pos, int pack) {
    const uint4 x = *reinterpret_cast<const uint4*>(src + pack * 8);
    const float* cs = p.cos_sin + pos * p.rot + pack * 4;
    const float4 c = __ldg(reinterpret_cast<const float4*>(cs));
    const float4 s = __ldg(reinterpret_cast<const float4*>(cs + half));
    auto turn = [](uint32_t uv, float co, float si) {
      const float u = bf16lo(uv), v = bf16hi(uv);
      return pack_bf16(u * co - v * si, v * co + u * si);
    };
    return make_uint4(turn(x.x, c.x, s.x), turn(x.y, c.y, s.y), turn(x.z, c.z, s.z),
                      turn(x.w, c.w, s.w));
  };
  auto position = [&](int64_t t) {
    int64_t pos = p.positions[t];
    if (pos < 0 || pos >= p.max_position) {
      if (p.status) atomicOr(p.status, FK_DEV_BAD_POSITION);
      pos = 0;
    }
    return pos;
  };
  if (blockIdx.x == 0) {
    const int from = p.copy ? 0 : p.q_rot_at >> 3;       // first pack written of a head
    const int packs = (p.q_out_pitch >> 3) - from;
    const int r0 = (p.q_rot_at >> 3) - from, r1 = r0 + (p.rot >> 3);
    for (int64_t t = blockIdx.y; t < p.rows; t += gridDim.y) {
      const int64_t pos = position(t);
      const uint16_t* q = static_cast<const uint16_t*>(p.q) + t * p.in_stride;
      uint16_t* out = static_cast<uint16_t*>(p.q_out) + t * p.heads * p.q_out_pitch;
      for (int i = threadIdx.x; i < p.heads * packs; i += blockDim.x) {
        const int h = i / packs, c = i - h * packs;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (c >= r0 && c < r1)
          v = rotated(q + h * p.q_pitch + p.dim, pos, c - r0);
        else if (p.copy && c * 8 < p.dim)
          v = *reinterpret_cast<const uint4*>(q + h * p.q_pitch + c * 8);
        *reinterpret_cast<uint4*>(out + h * p.q_out_pitch + (from + c) * 8) = v;
      }
    }
    return;
  }
  const int lane = threadIdx.x & 31;
  for (int64_t t = (int64_t)blockIdx.y * 8 + (threadIdx.x >> 5); t < p.rows;
       t += (int64_t)gridDim.y * 8) {
    const int64_t slot = p.slots[t];
    if (slot < 0 || slot >= p.num_slots) {
      if (slot >= p.num_slots && lane == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
      continue;
    }
    const int64_t pos = position(t);
    const uint16_t* src = static_cast<const uint16_t*>(p.lat) + t * p.in_stride;
    uint16_t* out = static_cast<uint16_t*>(p.cache) + slot * p.cache_pitch;
    constexpr int VPT = 4;                               // rank up to 1024
    uint4 x[VPT];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (lane + i * 32) * 8;
      x[i] = make_uint4(0u, 0u, 0u, 0u);
      if (c < p.rank) x[i] = *reinterpret_cast<const uint4*>(src + c);
      const uint32_t e[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += bf16lo(e[j]) * bf16lo(e[j]) + bf16hi(e[j]) * bf16hi(e[j]);
    }
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)p.rank + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (lane + i * 32) * 8;
      if (c >= p.rank) continue;
      const float4 a = __ldg(reinterpret_cast<const float4*>(p.weight + c));
      const float4 b = __ldg(reinterpret_cast<const float4*>(p.weight + c + 4));
      *reinterpret_cast<uint4*>(out + c) =
          make_uint4(pack_bf16(bf16lo(x[i].x) * rs * a.x, bf16hi(x[i].x) * rs * a.y),
                     pack_bf16(bf16lo(x[i].y) * rs * a.z, bf16hi(x[i].y) * rs * a.w),
                     pack_bf16(bf16lo(x[i].z) * rs * b.x, bf16hi(x[i].z) * rs * b.y),
                     pack_bf16(bf16lo(x[i].w) * rs * b.z, bf16hi(x[i].w) * rs * b.w));
    }
    for (int c = lane; c * 8 < p.cache_pitch - p.rank; c += 32)
      *reinterpret_cast<uint4*>(out + p.rank + c * 8) =
          c * 8 < p.rot ? rotated(src + p.rank, pos, c) : make_uint4(0u, 0u, 0u, 0u);
  }
}

__global__ void __launch_bounds__(256) latent_gather_kernel(
    const uint4* __restrict__ cache, int block_size, int num_blocks,
    const int32_t* __restrict__ block_tables, int64_t bt_stride, const int32_t* __restrict__ cu_k,
    int num_seqs, uint4* __restrict__ out, int64_t rows, int packs, int32_t* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  for (int64_t r = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5); r < rows;
       r += (int64_t)gridDim.x * 8) {
    int lo = 0, hi = num_seqs;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (cu_k[mid] <= r) lo = mid; else hi = mid;
    }
    const int key = (int)(r - cu_k[lo]);
    const int page = block_tables[lo * bt_stride + key / block_size];
    const bool ok = page >= 0 && page < num_blocks;
    if (!ok && lane == 0 && status) atomicOr(status, FK_DEV_BAD_PAGE);
    const uint4* src = cache + ((int64_t)(ok ? page : 0) * block_size + key % block_size) * packs;
    for (int c = lane; c < packs; c += 32)
      out[r * packs + c] = ok ? src[c] : make_uint4(0u, 0u, 0u, 0u);
  }
}

struct LatentAttnParams {
  const uint16_t* q; int64_t q_pitch;           // row (t * heads + h): q + row * q_pitch
  const uint16_t* cache; int cache_pitch;       // elements per cached row
  uint16_t* out; int64_t out_pitch;             // row (t * heads + h)
  float* part; float2* ml;                      // [splits][rows * heads][lo], (max, sum)
  const int32_t* cu_q; const int32_t* kv_lens;
  const int32_t* block_tables; int64_t bt_stride;
  int64_t flat_rows;                            // rows * heads
  int heads, lk, lo, block_size, num_blocks, splits, ring, run;
  float scale_log2;
  int32_t* status;
};

// Half of the warps make scores and softmax weights of a tile of 32 keys, the others multiply
// the weights of the tile before it with its values; one lane of them keeps the ring of tiles
// filled.  Latents up to 256 channels: 4 + 4 warps and two CTAs on an SM; above: 8 + 8 warps,
// scores of two tiles under way at once (SUBS = 2).  A tile is blocks of 64 channels, [32 rows][128 bytes] each, 128-byte swizzled by
// TMA.  The steps of a tile are short, so what bounds the kernel is the latency of fragment
// loads and of hand-overs: query fragments stay in registers, fragments are loaded several
// steps ahead, and warps hand over through named barriers (a wait on a shared-memory barrier
// costs several times as much; only the copies need one).
constexpr int LA_ROWS = 16, LA_KEYS = 32;
constexpr int LA_BLOCK = LA_KEYS * 128;
constexpr int LA_PPITCH = LA_KEYS + 8, LA_XPITCH = LA_KEYS + 8, LA_MAX_RING = 8;
constexpr uint32_t LA_WAIT_LIMIT = 1u << 22;
// named barriers
constexpr int LA_BAR_SUB = 1, LA_BAR_END = 3, LA_BAR_SUM = 4, LA_BAR_FULL = 5, LA_BAR_EMPTY = 7,
              LA_BAR_MAX = 9;

// lk: channels of a row, rounded up to 16; a tile holds whole blocks of 64.
__host__ __device__ constexpr int la_tile(int lk) { return (lk + 63) / 64 * LA_BLOCK; }
__host__ __device__ constexpr int la_subs(int rank) { return rank <= 256 ? 1 : 2; }
// 16-channel steps of scores per warp: registers for its part of the queries.
__host__ __device__ constexpr int la_steps(int rank) { return rank <= 128 ? 4 : rank <= 256 ? 6 : 10; }
__host__ __device__ constexpr int la_smem(int subs, int lk, int ring) {
  return ring * la_tile(lk) + subs * 4 * LA_ROWS * LA_XPITCH * 4 + 4 * LA_ROWS * LA_PPITCH * 2 +
         21 * LA_ROWS * 4 + LA_MAX_RING * 8 + 1024;
}
// Deepest ring that fits, 0: none.
__host__ __device__ constexpr int la_ring(int subs, int lk) {
  int r = LA_MAX_RING;
  while (r >= 3 && la_smem(subs, lk, r) > (subs == 1 ? 115712 : 232448)) --r;
  return r >= 3 ? r : 0;
}

__device__ __forceinline__ void named_bar_arrive(int id, int nthreads) {
  asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(nthreads) : "memory");
}

template <int RN, int QS, int SUBS>
__global__ void __launch_bounds__(SUBS * 256, 3 - SUBS)
latent_attn_kernel(const __grid_constant__ CUtensorMap tmap, const LatentAttnParams p) {
  extern __shared__ uint8_t la_raw[];
  constexpr int GROUP = SUBS * 128;                      // threads of either half
  pdl_launch_dependents();
  const int seq = blockIdx.y, split = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gr = lane >> 2, tq = lane & 3;
  uint8_t* K = la_raw + ((1024u - (smem_u32(la_raw) & 1023u)) & 1023u);    // ring of tiles
  const int tile_bytes = la_tile(p.lk);
  float* X = reinterpret_cast<float*>(K + p.ring * tile_bytes);   // [SUBS][4][16][LA_XPITCH]
  uint16_t* P = reinterpret_cast<uint16_t*>(X + SUBS * 4 * LA_ROWS * LA_XPITCH);  // [2][hi, lo][16][]
  float* alpha = reinterpret_cast<float*>(P + 4 * LA_ROWS * LA_PPITCH);    // [2][16]
  float* inv_l = alpha + 2 * LA_ROWS;                     // [16]
  float* m_run = inv_l + LA_ROWS;                         // [2][16]: running maximum
  float* m_warp = m_run + 2 * LA_ROWS;                    // [8][16]: of a tile, per warp
  float* l_warp = m_warp + 8 * LA_ROWS;                   // [8][16]
  uint64_t* full = reinterpret_cast<uint64_t*>(l_warp + 8 * LA_ROWS);      // [ring]
  if (tid == 0) {
    for (int i = 0; i < p.ring; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
    tma_prefetch_desc(&tmap);
  }
  pdl_wait();
  const int q0 = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q0;
  const int64_t first = (int64_t)q0 * p.heads + (int64_t)blockIdx.x * LA_ROWS;   // flat row
  const int64_t left = (int64_t)q_len * p.heads - (int64_t)blockIdx.x * LA_ROWS;
  if (left <= 0 || first + min(left, (int64_t)LA_ROWS) > p.flat_rows) return;
  const int n_rows = (int)min(left, (int64_t)LA_ROWS);
  const int kv_len = p.kv_lens[seq];
  const int before = kv_len - q_len + 1;                 // keys token 0 of the portion sees
  const int tok0 = blockIdx.x * LA_ROWS;
  const int most = max(0, min(kv_len, before + (tok0 + n_rows - 1) / p.heads));
  const int per = ((most + p.splits - 1) / p.splits + LA_KEYS - 1) / LA_KEYS * LA_KEYS;
  const int k_begin = min(most, split * per), k_end = min(most, k_begin + per);
  __syncthreads();
  const int tiles = (k_end - k_begin + LA_KEYS - 1) / LA_KEYS;
  // 16-byte chunk of a row's 128 bytes of a block, as the swizzle places it
  const int sw = lane & 7;
  const int row0 = gr, row1 = gr + 8;

  if (warp < GROUP / 32) {
    // --------------------------- scores and weights --------------------------
    // Four warps a tile.  With two tiles under way only the running maximum goes from one
    // tile to the next.  Products: a warp has all keys and a quarter of the channels.
    // Weights: 8 keys.
    constexpr int AHEAD = 3;
    const int sub = warp >> 2, v = warp & 3, key0 = v * 8;
    const int lim0 = row0 < n_rows ? min(k_end, before + (tok0 + row0) / p.heads) : 0;
    const int lim1 = row1 < n_rows ? min(k_end, before + (tok0 + row1) / p.heads) : 0;
    const int steps = p.lk >> 4, each = (steps + 3) >> 2;
    const int s0 = min(steps, v * each), s1 = min(steps, s0 + each);
    uint32_t qf[QS][4];
    {
      const uint16_t* r0 = p.q + (first + row0) * p.q_pitch + tq * 2;
      const uint16_t* r1 = p.q + (first + row1) * p.q_pitch + tq * 2;
#pragma unroll
      for (int u = 0; u < QS; ++u) {
        const int c = (s0 + u) * 16;
        const bool on = s0 + u < s1;
        qf[u][0] = on && row0 < n_rows ? *reinterpret_cast<const uint32_t*>(r0 + c) : 0u;
        qf[u][1] = on && row1 < n_rows ? *reinterpret_cast<const uint32_t*>(r1 + c) : 0u;
        qf[u][2] = on && row0 < n_rows ? *reinterpret_cast<const uint32_t*>(r0 + c + 8) : 0u;
        qf[u][3] = on && row1 < n_rows ? *reinterpret_cast<const uint32_t*>(r1 + c + 8) : 0u;
      }
    }
    const int krow = (lane & 7) + (lane >> 4) * 8, khi = (lane >> 3) & 1;
    float* xs = X + sub * 4 * LA_ROWS * LA_XPITCH;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    bool ok = true;
    int st = sub;
    uint32_t phase = 0;
    for (int n = sub; n < tiles; n += SUBS) {
      const int buf = n & 1;
      const int k0 = k_begin + n * LA_KEYS;
      ok = ok && mbar_wait(&full[st], phase, LA_WAIT_LIMIT);
      uint8_t* tile = K + st * tile_bytes;
      if (k0 + LA_KEYS > k_end) {
        // rows behind the last key belong to nobody: their weights are zero, and so must
        // the products be
        const int per_row = tile_bytes / (LA_KEYS * 16);
        for (int i = tid & 127; i < (k0 + LA_KEYS - k_end) * per_row; i += 128) {
          const int r = k_end - k0 + i / per_row, c = i % per_row;
          *reinterpret_cast<uint4*>(tile + (c >> 3) * LA_BLOCK + r * 128 + (c & 7) * 16) =
              make_uint4(0u, 0u, 0u, 0u);
        }
        named_bar_sync(LA_BAR_SUB + sub, 128);
      }
      const uint32_t ka = smem_u32(tile) + krow * 128;
      float s[4][4] = {};
      uint32_t b[AHEAD + 1][2][4];
      auto load = [&](int u, uint32_t (&fb)[2][4]) {
        const int i = min(s0 + u, steps - 1);
        const uint32_t at = ka + (i >> 2) * LA_BLOCK + ((((i & 3) * 2 + khi) ^ sw) << 4);
        ldmatrix_x4(at, fb[0][0], fb[0][1], fb[0][2], fb[0][3]);
        ldmatrix_x4(at + 16 * 128, fb[1][0], fb[1][1], fb[1][2], fb[1][3]);
      };
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) load(u, b[u]);
#pragma unroll
      for (int u = 0; u < QS; ++u) {
        if (u + AHEAD < QS) load(u + AHEAD, b[(u + AHEAD) % (AHEAD + 1)]);
        const uint32_t (&fb)[2][4] = b[u % (AHEAD + 1)];
        // steps beyond the part have zero queries
        mma_bf16_16816(s[0], qf[u], fb[0][0], fb[0][1]);
        mma_bf16_16816(s[1], qf[u], fb[0][2], fb[0][3]);
        mma_bf16_16816(s[2], qf[u], fb[1][0], fb[1][1]);
        mma_bf16_16816(s[3], qf[u], fb[1][2], fb[1][3]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          *reinterpret_cast<float2*>(xs + (v * LA_ROWS + row0 + e * 8) * LA_XPITCH + j * 8 +
                                     tq * 2) = make_float2(s[j][e * 2], s[j][e * 2 + 1]);
      named_bar_sync(LA_BAR_SUB + sub, 128);
      float x[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int q = 0; q < 4; ++q)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 y = *reinterpret_cast<const float2*>(
              xs + (q * LA_ROWS + row0 + e * 8) * LA_XPITCH + key0 + tq * 2);
          x[e * 2] += y.x;
          x[e * 2 + 1] += y.y;
        }
      float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = k0 + key0 + tq * 2 + e;
        x[e] = key < lim0 ? x[e] * p.scale_log2 : -INFINITY;
        x[2 + e] = key < lim1 ? x[2 + e] * p.scale_log2 : -INFINITY;
        t0 = fmaxf(t0, x[e]);
        t1 = fmaxf(t1, x[2 + e]);
      }
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, o));
        t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, o));
      }
      if (tq == 0) {
        m_warp[warp * LA_ROWS + row0] = t0;
        m_warp[warp * LA_ROWS + row1] = t1;
      }
      named_bar_sync(LA_BAR_SUB + sub, 128);
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float* mw = m_warp + (sub * 4 + w) * LA_ROWS;
        t0 = fmaxf(t0, mw[row0]);
        t1 = fmaxf(t1, mw[row1]);
      }
      float p0 = m0, p1 = m1;
      if (SUBS == 2 && n > 0) {
        named_bar_sync(LA_BAR_MAX + (sub ^ 1), 2 * 128);
        p0 = m_run[(sub ^ 1) * LA_ROWS + row0];
        p1 = m_run[(sub ^ 1) * LA_ROWS + row1];
      }
      t0 = fmaxf(t0, p0);
      t1 = fmaxf(t1, p1);
      const bool writes = tq == 0 && v == 0;
      if (writes) {
        m_run[sub * LA_ROWS + row0] = t0;
        m_run[sub * LA_ROWS + row1] = t1;
      }
      if (SUBS == 2 && n + 1 < tiles) named_bar_arrive(LA_BAR_MAX + sub, 2 * 128);
      const float z0 = t0 == -INFINITY ? 0.f : t0, z1 = t1 == -INFINITY ? 0.f : t1;
      l0 *= fast_exp2(m0 - z0);
      l1 *= fast_exp2(m1 - z1);
      m0 = t0;
      m1 = t1;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        x[e] = fast_exp2(x[e] - z0);
        x[2 + e] = fast_exp2(x[2 + e] - z1);
        l0 += x[e];
        l1 += x[2 + e];
      }
      if (n >= 2) named_bar_sync(LA_BAR_EMPTY + buf, 128 + GROUP);
      uint16_t* ph = P + buf * 2 * LA_ROWS * LA_PPITCH + key0 + tq * 2;
      uint32_t hi, lo;
      split_bf16(x[0], x[1], &hi, &lo);
      *reinterpret_cast<uint32_t*>(ph + row0 * LA_PPITCH) = hi;
      *reinterpret_cast<uint32_t*>(ph + (LA_ROWS + row0) * LA_PPITCH) = lo;
      split_bf16(x[2], x[3], &hi, &lo);
      *reinterpret_cast<uint32_t*>(ph + row1 * LA_PPITCH) = hi;
      *reinterpret_cast<uint32_t*>(ph + (LA_ROWS + row1) * LA_PPITCH) = lo;
      if (writes) {
        alpha[buf * LA_ROWS + row0] = p0 == -INFINITY ? 1.f : fast_exp2(p0 - z0);
        alpha[buf * LA_ROWS + row1] = p1 == -INFINITY ? 1.f : fast_exp2(p1 - z1);
      }
      named_bar_arrive(LA_BAR_FULL + buf, 128 + GROUP);
      st += SUBS;
      if (st >= p.ring) { st -= p.ring; phase ^= 1; }
    }
    if (!ok && p.status) atomicOr(p.status, FK_DEV_WAIT_TIMEOUT);
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      l0 += __shfl_xor_sync(0xffffffffu, l0, o);
      l1 += __shfl_xor_sync(0xffffffffu, l1, o);
    }
    // sums relative to the last maximum this warp has seen
    if (tq == 0) {
      l_warp[warp * LA_ROWS + row0] = l0;
      l_warp[warp * LA_ROWS + row1] = l1;
    }
    if (tiles <= sub && v == 0 && lane < LA_ROWS) m_run[sub * LA_ROWS + lane] = -INFINITY;
    named_bar_sync(LA_BAR_SUM, GROUP);
    if (tid < LA_ROWS) {
      const float ma = m_run[tid], mb = SUBS == 2 ? m_run[LA_ROWS + tid] : ma;
      const float mx = fmaxf(ma, mb);
      const float z = mx == -INFINITY ? 0.f : mx;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < 4 * SUBS; ++w)
        l += l_warp[w * LA_ROWS + tid] * fast_exp2((w < 4 ? ma : mb) - z);
      inv_l[tid] = l > 0.f ? 1.0f / l : 0.f;
      if (p.splits > 1 && tid < n_rows)
        p.ml[(int64_t)split * p.flat_rows + first + tid] = make_float2(mx, l);
    }
    named_bar_sync(LA_BAR_END, 2 * GROUP);
    return;
  }

  // -------------------------------- values ---------------------------------
  // The ring: tile n comes into slot n % ring.  When the weights of tile n have been handed
  // over, every warp here is through with tile n - 1: its slot takes the next tile.
  const int32_t* bt = p.block_tables + seq * p.bt_stride;
  // row of the pool where the run of keys from `key` on begins; out of range: zeros
  auto pool_row = [&](int key) {
    const int none = p.num_blocks * p.block_size;
    if (key >= k_end) return none;
    const int page = bt[key / p.block_size];
    if (page >= 0 && page < p.num_blocks) return page * p.block_size + key % p.block_size;
    if (p.status) atomicOr(p.status, FK_DEV_BAD_PAGE);
    return none;
  };
  auto issue = [&](int n, int slot, int first_row) {
    mbar_arrive_expect_tx(&full[slot], (uint32_t)tile_bytes);
    uint8_t* dst = K + slot * tile_bytes;
    if (p.run == LA_KEYS) {
      tma_load_3d(dst, &tmap, &full[slot], 0, first_row, 0);    // the whole tile
    } else {
      // runs of p.run keys lie in one page; blocks of 64 channels one by one
      for (int r = 0; r < LA_KEYS; r += p.run) {
        const int row = r == 0 ? first_row : pool_row(k_begin + n * LA_KEYS + r);
        for (int c = 0; c < tile_bytes / LA_BLOCK; ++c)
          tma_load_3d(dst + c * LA_BLOCK + r * 128, &tmap, &full[slot], 0, row, c);
      }
    }
  };
  const bool feeds = warp == GROUP / 32 && lane == 0;
  int next_row = 0;                       // of tile n - 1 + ring, looked up ahead
  if (feeds) {
    for (int n = 0; n < min(tiles, p.ring); ++n) issue(n, n, pool_row(k_begin + n * LA_KEYS));
    if (tiles > p.ring) next_row = pool_row(k_begin + p.ring * LA_KEYS);
  }
  __syncwarp();
  float acc[RN][4];
#pragma unroll
  for (int j = 0; j < RN; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
  const int col0 = (warp - GROUP / 32) * RN * 8;
  uint32_t at[RN / 2];                    // this lane's fragment addresses inside a tile
#pragma unroll
  for (int j = 0; j < RN / 2; ++j) {
    // columns beyond the latent are not stored: any column of the row will do
    const int c = min(col0 + j * 16, p.lo - 16);
    at[j] = (lane & 15) * 128 + (c >> 6) * LA_BLOCK + ((((c >> 3) & 7) + (lane >> 4)) ^ sw) * 16;
  }
  const uint32_t pa = smem_u32(P + (lane & 15) * LA_PPITCH + (lane >> 4) * 8);
  int st = 0;
  for (int n = 0; n < tiles; ++n) {
    const int buf = n & 1;
    const uint32_t tile = smem_u32(K) + st * tile_bytes;
    named_bar_sync(LA_BAR_FULL + buf, 128 + GROUP);
    if (feeds && n > 0 && n - 1 + p.ring < tiles) {
      issue(n - 1 + p.ring, st == 0 ? p.ring - 1 : st - 1, next_row);
      if (n + p.ring < tiles) next_row = pool_row(k_begin + (n + p.ring) * LA_KEYS);
    }
    __syncwarp();
    if (col0 < p.lo) {
      uint32_t ph[2][4], pl[2][4], b[2][RN / 2][4];
      const uint32_t pb = pa + buf * 2 * LA_ROWS * LA_PPITCH * 2;
#pragma unroll
      for (int kt = 0; kt < 2; ++kt) {
        ldmatrix_x4(pb + kt * 32, ph[kt][0], ph[kt][1], ph[kt][2], ph[kt][3]);
        ldmatrix_x4(pb + kt * 32 + LA_ROWS * LA_PPITCH * 2, pl[kt][0], pl[kt][1], pl[kt][2],
                    pl[kt][3]);
#pragma unroll
        for (int j = 0; j < RN / 2; ++j)
          ldmatrix_x4_trans(tile + kt * 16 * 128 + at[j], b[kt][j][0], b[kt][j][1], b[kt][j][2],
                            b[kt][j][3]);
      }
      const float a0 = alpha[buf * LA_ROWS + row0], a1 = alpha[buf * LA_ROWS + row1];
      if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
        for (int j = 0; j < RN; ++j) {
          acc[j][0] *= a0; acc[j][1] *= a0;
          acc[j][2] *= a1; acc[j][3] *= a1;
        }
      }
#pragma unroll
      for (int kt = 0; kt < 2; ++kt)
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int j = 0; j < RN / 2; ++j) {
            mma_bf16_16816(acc[2 * j], part ? pl[kt] : ph[kt], b[kt][j][0], b[kt][j][1]);
            mma_bf16_16816(acc[2 * j + 1], part ? pl[kt] : ph[kt], b[kt][j][2], b[kt][j][3]);
          }
    }
    if (n + 2 < tiles) named_bar_arrive(LA_BAR_EMPTY + buf, 128 + GROUP);
    if (++st == p.ring) st = 0;
  }
  named_bar_sync(LA_BAR_END, 2 * GROUP);
  if (p.splits > 1 && tiles == 0) return;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = gr + e * 8;
    if (r >= n_rows) continue;
    if (p.splits > 1) {
      float* o = p.part + ((int64_t)split * p.flat_rows + first + r) * p.lo;
#pragma unroll
      for (int j = 0; j < RN; ++j) {
        const int c = col0 + j * 8 + tq * 2;
        if (c < p.lo)
          *reinterpret_cast<float2*>(o + c) = make_float2(acc[j][e * 2], acc[j][e * 2 + 1]);
      }
    } else {
      const float inv = inv_l[r];
      uint16_t* o = p.out + (first + r) * p.out_pitch;
#pragma unroll
      for (int j = 0; j < RN; ++j) {
        const int c = col0 + j * 8 + tq * 2;
        if (c < p.lo)
          *reinterpret_cast<uint32_t*>(o + c) =
              pack_bf16(acc[j][e * 2] * inv, acc[j][e * 2 + 1] * inv);
      }
    }
  }
}

// One CTA per (token, head) row; at most 32 ranges, a lane each.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float share[32];
  const int64_t r = blockIdx.x;
  if (threadIdx.x < 32) {
    const int s = threadIdx.x;
    const float2 v = s < p.splits ? p.ml[(int64_t)s * p.flat_rows + r] : make_float2(0.f, 0.f);
    const bool on = v.y > 0.f;
    float mx = on ? v.x : -INFINITY;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float w = on ? exp2f(v.x - mx) : 0.f;
    const float l = warp_sum(w * v.y);
    share[s] = l > 0.f ? w / l : 0.f;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < p.lo; c += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float w = share[s];
      if (w > 0.f)
        a = a + *reinterpret_cast<const float4*>(
                    p.part + ((int64_t)s * p.flat_rows + r) * p.lo + c) * w;
    }
    Elem<uint16_t>::store4(p.out + r * p.out_pitch + c, a);
  }
}

// [rows, channels] bf16 pool as (64 channels, rows, blocks of 64 channels): box = `run` rows
// of `blocks` blocks, 128B swizzle
static int la_map(const void* ptr, int64_t rows, int64_t cols, int run, int blocks,
                  CUtensorMap* out) {
  struct Entry { const void* ptr; int64_t rows, cols; int run, blocks; CUtensorMap map; };
  static std::mutex mu;
  static std::vector<Entry> maps;
  std::lock_guard<std::mutex> lk(mu);
  for (const Entry& e : maps)
    if (e.ptr == ptr && e.rows == rows && e.cols == cols && e.run == run &&
        e.blocks == blocks) {
      *out = e.map;
      return FK_OK;
    }
  tensormap_encode_fn enc = get_tensormap_encode();
  FK_REQUIRE(enc != nullptr, FK_ERR_CUDA,
             "cuTensorMapEncodeTiled not available from the driver");
  cuuint64_t dims[3] = {64, (cuuint64_t)rows, (cuuint64_t)(cols / 64)};
  cuuint64_t strides[2] = {(cuuint64_t)cols * 2, 128};
  cuuint32_t box[3] = {64, (cuuint32_t)run, (cuuint32_t)blocks};
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims,
                   strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  FK_REQUIRE(r == CUDA_SUCCESS, FK_ERR_CUDA, "cuTensorMapEncodeTiled failed with code %d",
             (int)r);
  if (maps.size() > 1024) maps.clear();
  maps.push_back({ptr, rows, cols, run, blocks, *out});
  return FK_OK;
}

template <int RN, int QS, int SUBS>
static int launch_latent(LatentAttnParams& p, dim3 grid, cudaStream_t s) {
  p.ring = la_ring(SUBS, p.lk);
  const int smem = la_smem(SUBS, p.lk, p.ring);
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, latent_attn_kernel<RN, QS, SUBS>,
                                  SUBS == 1 ? 115712 : 232448));
  p.run = LA_KEYS;                       // keys that surely lie in one page
  while (p.block_size % p.run) p.run /= 2;
  CUtensorMap map;
  const int rc = la_map(p.cache, (int64_t)p.num_blocks * p.block_size, p.cache_pitch, p.run,
                        p.run == LA_KEYS ? (p.lk + 63) / 64 : 1, &map);
  if (rc != FK_OK) return rc;
  FK_CUDA_OK(launch_kernel(latent_attn_kernel<RN, QS, SUBS>, grid, dim3(SUBS * 256),
                           (size_t)smem, s, map, p));
  count_launch();
  return FK_OK;
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_latent_prepare(const void* q, const void* latent, int64_t in_stride, int q_pitch,
                      int is_f32, const float* weight, const float* cos_sin, int64_t max_position,
                      const int32_t* slots, const int64_t* positions, void* cache,
                      int64_t num_slots, int cache_pitch, void* q_out, int q_out_pitch,
                      int q_rot_at, int copy, int64_t rows, int heads, int dim, int rot, int rank,
                      float eps, int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && heads > 0 && dim > 0 && rot >= 0 && rot % 2 == 0 && rank > 0,
             FK_ERR_INVALID_ARG, "fk_latent_prepare: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(q && latent && weight && cos_sin && slots && positions && cache && q_out,
             FK_ERR_INVALID_ARG, "fk_latent_prepare: null pointer");
  FK_REQUIRE(q_pitch >= dim + rot && cache_pitch >= rank + rot && q_out_pitch >= q_rot_at + rot &&
                 q_rot_at >= 0 && (!copy || q_rot_at >= dim),
             FK_ERR_INVALID_ARG, "fk_latent_prepare: bad layout");
  LatentPrepParams p{};
  p.q = q; p.lat = latent; p.in_stride = in_stride; p.q_pitch = q_pitch; p.weight = weight;
  p.cos_sin = cos_sin; p.max_position = max_position; p.slots = slots; p.positions = positions;
  p.cache = cache; p.num_slots = num_slots; p.cache_pitch = cache_pitch; p.q_out = q_out;
  p.q_out_pitch = q_out_pitch; p.q_rot_at = q_rot_at; p.copy = copy; p.rows = rows;
  p.heads = heads; p.dim = dim; p.rot = rot; p.rank = rank; p.eps = eps; p.status = status;
  const dim3 grid((unsigned)((heads + 1 + 7) / 8), (unsigned)(rows < 16384 ? rows : 16384));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = !is_f32 && rank <= 1024 &&
                   (dim | rot | rank | q_pitch | cache_pitch | q_out_pitch | q_rot_at) % 8 == 0 &&
                   in_stride % 8 == 0 && aligned16(q) && aligned16(latent) && aligned16(weight) &&
                   aligned16(cos_sin) && aligned16(cache) && aligned16(q_out);
  if (vec) {
    const dim3 vgrid(2, (unsigned)(rows < 16384 ? rows : 16384));
    FK_CUDA_OK(launch_kernel(latent_prepare_vec_kernel, vgrid, dim3(256), 0, s, p));
    count_launch();
    return FK_OK;
  }
  FK_CUDA_OK(is_f32 ? launch_kernel(latent_prepare_kernel<float>, grid, dim3(256), 0, s, p)
                    : launch_kernel(latent_prepare_kernel<uint16_t>, grid, dim3(256), 0, s, p));
  count_launch();
  return FK_OK;
}

int fk_latent_gather(const void* cache, int64_t row_bytes, int64_t num_blocks, int block_size,
                     const int32_t* block_tables, int64_t block_table_stride,
                     const int32_t* cu_seqlens_k, int num_seqs, void* out, int64_t rows,
                     int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && num_seqs >= 0 && block_size > 0 && num_blocks > 0,
             FK_ERR_INVALID_ARG, "fk_latent_gather: bad sizes");
  if (rows == 0 || num_seqs == 0) return FK_OK;
  FK_REQUIRE(cache && block_tables && cu_seqlens_k && out, FK_ERR_INVALID_ARG,
             "fk_latent_gather: null pointer");
  FK_REQUIRE(row_bytes > 0 && row_bytes % 16 == 0 && aligned16(cache) && aligned16(out),
             FK_ERR_ALIGNMENT, "fk_latent_gather: rows must be 16-byte aligned");
  const int64_t want = (rows + 7) / 8, cap = (int64_t)sm_count() * 16;
  FK_CUDA_OK(launch_kernel(latent_gather_kernel, dim3((unsigned)(want < cap ? want : cap)),
                           dim3(256), 0, static_cast<cudaStream_t>(stream), (const uint4*)cache,
                           block_size, (int)num_blocks, block_tables, block_table_stride,
                           cu_seqlens_k, num_seqs, (uint4*)out, rows, (int)(row_bytes / 16),
                           status));
  count_launch();
  return FK_OK;
}

int fk_latent_attn_supported(int rank, int rot) {
  const int lk = (rank + rot + 15) / 16 * 16;
  return rank > 0 && rank <= 512 && rot >= 0 && lk / 16 <= 4 * la_steps(rank) &&
         la_ring(la_subs(rank), lk) > 0;
}

/* Key ranges a call with these sizes splits its rows into.  The lengths are on the device, so
 * 2048 keys stand for them: the number with the shortest rounds of CTAs, each with its share
 * of the keys and a start that costs as much as about 256. */
int fk_latent_attn_splits(int num_seqs, int64_t max_q, int heads, int rank, int64_t max_keys) {
  const int64_t tiles = (max_q * heads + LA_ROWS - 1) / LA_ROWS * num_seqs;
  const int64_t slots = (int64_t)sm_count() * (la_subs(rank) == 1 ? 2 : 1);
  const int64_t keys = max_keys < 2048 ? max_keys : 2048;
  int best = 1;
  int64_t best_cost = INT64_MAX;
  for (int s = 1; s <= 32 && (s == 1 || s * 128 <= max_keys + 127); ++s) {
    const int64_t cost = (tiles * s + slots - 1) / slots * ((keys + s - 1) / s + 256);
    if (cost < best_cost) { best = s; best_cost = cost; }
  }
  return best;
}

int64_t fk_latent_attn_workspace_floats(int64_t rows, int heads, int rank, int splits) {
  return splits <= 1 ? 0 : (int64_t)splits * rows * heads * ((rank + 15) / 16 * 16 + 2);
}

int fk_latent_attn(const void* q, int64_t q_pitch, const void* cache, int64_t num_blocks,
                   int block_size, int cache_pitch, void* out, int64_t out_pitch,
                   const int32_t* cu_seqlens_q, const int32_t* kv_lens,
                   const int32_t* block_tables, int64_t block_table_stride, int num_seqs,
                   int64_t rows, int64_t max_seqlen_q, int heads, int rank, int rot,
                   float softmax_scale, int splits, float* workspace, int64_t workspace_floats,
                   int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && num_seqs >= 0 && heads > 0 && rank > 0 && rot >= 0 && splits >= 1 &&
                 splits <= 32,
             FK_ERR_INVALID_ARG, "fk_latent_attn: bad sizes");
  if (rows == 0 || num_seqs == 0 || max_seqlen_q <= 0) return FK_OK;
  FK_REQUIRE(q && cache && out && cu_seqlens_q && kv_lens && block_tables, FK_ERR_INVALID_ARG,
             "fk_latent_attn: null pointer");
  FK_REQUIRE(fk_latent_attn_supported(rank, rot), FK_ERR_UNSUPPORTED,
             "fk_latent_attn: rank %d with %d rotated channels", rank, rot);
  const int lk = (rank + rot + 15) / 16 * 16, lo = (rank + 15) / 16 * 16;
  FK_REQUIRE(cache_pitch % 64 == 0, FK_ERR_UNSUPPORTED,
             "fk_latent_attn: cached rows of %d elements, not a multiple of 64", cache_pitch);
  FK_REQUIRE(cache_pitch >= lk && q_pitch >= lk && out_pitch >= lo && block_size > 0 &&
                 num_blocks > 0 && num_blocks * block_size < (1ll << 31),
             FK_ERR_INVALID_ARG, "fk_latent_attn: rows shorter than latent and rotated key, "
             "rounded up to 16 elements");
  FK_REQUIRE(block_size % 8 == 0, FK_ERR_UNSUPPORTED,
             "fk_latent_attn: block_size %d must be a multiple of 8", block_size);
  FK_REQUIRE(cache_pitch % 8 == 0 && q_pitch % 8 == 0 && out_pitch % 4 == 0 && aligned16(q) &&
                 aligned16(cache) && aligned16(out) && aligned16(workspace),
             FK_ERR_ALIGNMENT, "fk_latent_attn: rows must be 16-byte aligned");
  FK_REQUIRE(splits == 1 || (workspace && workspace_floats >=
                             fk_latent_attn_workspace_floats(rows, heads, rank, splits)),
             FK_ERR_WORKSPACE, "fk_latent_attn: workspace too small");
  LatentAttnParams p{};
  p.q = static_cast<const uint16_t*>(q); p.q_pitch = q_pitch;
  p.cache = static_cast<const uint16_t*>(cache); p.cache_pitch = cache_pitch;
  p.out = static_cast<uint16_t*>(out); p.out_pitch = out_pitch;
  p.flat_rows = rows * heads;
  p.part = workspace;
  p.ml = workspace ? reinterpret_cast<float2*>(workspace + (int64_t)splits * p.flat_rows * lo)
                   : nullptr;
  p.cu_q = cu_seqlens_q; p.kv_lens = kv_lens; p.block_tables = block_tables;
  p.bt_stride = block_table_stride; p.heads = heads; p.lk = lk; p.lo = lo;
  p.block_size = block_size; p.num_blocks = (int)num_blocks; p.splits = splits;
  p.scale_log2 = softmax_scale * 1.4426950408889634f; p.status = status;
  const int64_t tiles = (max_seqlen_q * heads + LA_ROWS - 1) / LA_ROWS;
  FK_REQUIRE(tiles <= 0x7fffffff && num_seqs <= 65535 && p.flat_rows <= 0x7fffffff,
             FK_ERR_UNSUPPORTED, "fk_latent_attn: too many rows");
  const dim3 grid((unsigned)tiles, (unsigned)num_seqs, (unsigned)splits);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int rc = rank <= 128   ? launch_latent<4, la_steps(128), 1>(p, grid, s)
                 : rank <= 256 ? launch_latent<8, la_steps(256), 1>(p, grid, s)
                               : launch_latent<8, la_steps(512), 2>(p, grid, s);
  if (rc != FK_OK || splits == 1) return rc;
  FK_CUDA_OK(launch_kernel(latent_merge_kernel, dim3((unsigned)p.flat_rows), dim3(128), 0, s, p));
  count_launch();
  return FK_OK;
}

}  // extern "C"
