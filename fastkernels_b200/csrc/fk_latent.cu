// Latent attention: one cached row per token, [latent (rank) | rotated key (rot)], shared by
// all heads.  With the key and value projections of a head taken into its query and its
// output ("absorbed"), a head's query is [W_uk^T q | rotated q], its keys are the cached rows
// and its values the first `rank` channels of them.
//
//   latent_prepare_kernel   norm of the latent, rotation of the shared key, store; rotation
//                           (and copy) of the queries; _vec: the same 16 bytes at a time
//   latent_gather_kernel    cached rows of a batch's sequences side by side
//   latent_attn_kernel      absorbed attention, bf16: portions and single tokens alike.  A
//                           CTA owns HT (token, head) rows of one sequence and a range of
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

// Warps 0-7 make scores and softmax weights of a tile of 32 keys, warps 8-15 multiply the
// weights of the tile before it with its values, warp 16 keeps the ring of tiles filled: a
// tile is blocks of 64 channels, [32 rows][128 bytes] each, 128-byte swizzled by TMA.
constexpr int LA_GROUP = 256, LA_THREADS = 2 * LA_GROUP + 32, LA_KEYS = 32;
constexpr int LA_BLOCK = LA_KEYS * 128;
constexpr int LA_PPITCH = LA_KEYS + 8, LA_MAX_RING = 8;
constexpr uint32_t LA_WAIT_LIMIT = 1u << 22;

// lk: channels of a row, rounded up to 16; a tile holds whole blocks of 64.
__host__ __device__ constexpr int la_tile(int lk) { return (lk + 63) / 64 * LA_BLOCK; }
__host__ __device__ constexpr int la_smem(int ht, int lk, int ring) {
  return ring * la_tile(lk) + ht * (lk + 8) * 2 + 4 * ht * LA_PPITCH * 2 + 21 * ht * 4 +
         (2 * LA_MAX_RING + 6) * 8 + 1024;
}
// Deepest ring that fits, 0: none.
__host__ __device__ constexpr int la_ring(int ht, int lk) {
  int r = LA_MAX_RING;
  while (r >= 3 && la_smem(ht, lk, r) > 232448) --r;
  return r >= 3 ? r : 0;
}

template <int HT, int RN>
__global__ void __launch_bounds__(LA_THREADS, 1)
latent_attn_kernel(const __grid_constant__ CUtensorMap tmap, const LatentAttnParams p) {
  extern __shared__ uint8_t la_raw[];
  pdl_launch_dependents();
  constexpr int MTS = HT / 16;
  const int seq = blockIdx.y, split = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gr = lane >> 2, tq = lane & 3;
  uint8_t* K = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(la_raw) + 1023) &
                                          ~uintptr_t(1023));          // ring of tiles
  const int tile_bytes = la_tile(p.lk), kp = p.lk + 8;
  uint16_t* Q = reinterpret_cast<uint16_t*>(K + p.ring * tile_bytes); // [HT][kp]
  uint16_t* P = Q + HT * kp;                              // [2][hi, lo][HT][LA_PPITCH]
  float* alpha = reinterpret_cast<float*>(P + 4 * HT * LA_PPITCH);    // [2][HT]
  float* inv_l = alpha + 2 * HT;                          // [HT]
  float* m_run = inv_l + HT;                              // [2][HT]: running maximum
  float* m_warp = m_run + 2 * HT;                         // [8][HT]: of a tile, per warp
  float* l_warp = m_warp + 8 * HT;                        // [8][HT]
  uint64_t* full = reinterpret_cast<uint64_t*>(l_warp + 8 * HT);   // [ring]: rows have come
  uint64_t* empty = full + LA_MAX_RING;                   // [ring]: ... and are no longer read
  uint64_t* p_full = empty + LA_MAX_RING;                 // [2]: weights of a tile written
  uint64_t* p_empty = p_full + 2;                         // [2]: ... and read
  uint64_t* m_full = p_empty + 2;                         // [2]: running maximum after a tile
  if (tid == 0) {
    for (int i = 0; i < p.ring; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], LA_GROUP / 32);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&p_full[i], 4);
      mbar_init(&p_empty[i], LA_GROUP / 32);
      mbar_init(&m_full[i], 4);
    }
    mbar_fence_init();
    tma_prefetch_desc(&tmap);
  }
  pdl_wait();
  const int q0 = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q0;
  const int64_t first = (int64_t)q0 * p.heads + (int64_t)blockIdx.x * HT;   // flat row
  const int64_t left = (int64_t)q_len * p.heads - (int64_t)blockIdx.x * HT;
  if (left <= 0 || first + min(left, (int64_t)HT) > p.flat_rows) return;
  const int n_rows = (int)min(left, (int64_t)HT);
  const int kv_len = p.kv_lens[seq];
  const int before = kv_len - q_len + 1;                 // keys token 0 of the portion sees
  const int tok0 = blockIdx.x * HT;
  const int most = max(0, min(kv_len, before + (tok0 + n_rows - 1) / p.heads));
  const int per = ((most + p.splits - 1) / p.splits + LA_KEYS - 1) / LA_KEYS * LA_KEYS;
  const int k_begin = min(most, split * per), k_end = min(most, k_begin + per);
  {
    const int packs = p.lk >> 3;
    for (int i = tid; i < HT * packs; i += LA_THREADS) {
      const int r = i / packs, c = (i - r * packs) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < n_rows) v = *reinterpret_cast<const uint4*>(p.q + (first + r) * p.q_pitch + c);
      *reinterpret_cast<uint4*>(Q + r * kp + c) = v;
    }
  }
  __syncthreads();
  const int tiles = (k_end - k_begin + LA_KEYS - 1) / LA_KEYS;
  bool ok = true;

  if (warp == 2 * LA_GROUP / 32) {
    // ------------------------------- cached rows ----------------------------
    if (lane != 0) return;
    const int32_t* bt = p.block_tables + seq * p.bt_stride;
    const int blocks = (p.lk + 63) / 64;
    int n = 0;
    for (; n < tiles; ++n) {
      const int st = n % p.ring;
      if (n >= p.ring)
        ok = mbar_wait(&empty[st], (uint32_t)(n / p.ring - 1) & 1u, LA_WAIT_LIMIT);
      if (!ok) {
        if (p.status) atomicOr(p.status, FK_DEV_WAIT_TIMEOUT);
        break;
      }
      mbar_arrive_expect_tx(&full[st], (uint32_t)tile_bytes);
      uint8_t* dst = K + st * tile_bytes;
      // runs of p.run keys lie in one page
      for (int r = 0; r < LA_KEYS; r += p.run) {
        const int key = k_begin + n * LA_KEYS + r;
        int row = p.num_blocks * p.block_size;            // out of range: zeros
        if (key < k_end) {
          const int page = bt[key / p.block_size];
          if (page >= 0 && page < p.num_blocks) row = page * p.block_size + key % p.block_size;
          else if (p.status) atomicOr(p.status, FK_DEV_BAD_PAGE);
        }
        for (int c = 0; c < blocks; ++c)
          tma_load_2d(dst + c * LA_BLOCK + r * 128, &tmap, &full[st], c * 64, row);
      }
    }
    // no copy may be in flight when the CTA ends
    if (!ok)
      for (int i = max(0, n - p.ring); i < n; ++i)
        (void)mbar_wait(&full[i % p.ring], (uint32_t)(i / p.ring) & 1u, LA_WAIT_LIMIT);
    return;
  }

  // 16-byte chunk of a row's 128 bytes of a block, as the swizzle places it
  const int sw = lane & 7;

  if (warp < LA_GROUP / 32) {
    // --------------------------- scores and weights --------------------------
    // Four warps a tile, so that two tiles are under way; only the running maximum goes from
    // one tile to the next.  HT = 16: a warp takes 8 keys.  HT = 32: 16 rows by 16 keys.
    constexpr int NK = MTS;                        // 8-key groups of a warp
    const int sub = warp >> 2, v = warp & 3;
    const int mt = MTS == 2 ? v & 1 : 0, key0 = MTS == 2 ? (v >> 1) * 16 : v * 8;
    const int row0 = mt * 16 + gr, row1 = row0 + 8;
    const int lim0 = row0 < n_rows ? min(k_end, before + (tok0 + row0) / p.heads) : 0;
    const int lim1 = row1 < n_rows ? min(k_end, before + (tok0 + row1) / p.heads) : 0;
    const int steps = p.lk >> 4;
    const uint32_t qa = smem_u32(Q + (mt * 16 + (lane & 15)) * kp + (lane >> 4) * 8);
    // HT = 16: 8 keys by 32 channels a load, HT = 32: 16 keys by 16
    const int krow = MTS == 2 ? key0 + (lane & 7) + (lane >> 4) * 8 : key0 + (lane & 7);
    const int khi = MTS == 2 ? (lane >> 3) & 1 : lane >> 3;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    for (int n = sub; n < tiles; n += 2) {
      const int k0 = k_begin + n * LA_KEYS, st = n % p.ring;
      ok = ok && mbar_wait(&full[st], (uint32_t)(n / p.ring) & 1u, LA_WAIT_LIMIT);
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
        named_bar_sync(1 + sub, 128);
      }
      const uint32_t ka = smem_u32(tile) + krow * 128;
      float s[2][NK][4] = {};                      // two chains of products
      // fragments of UN steps come ahead of the products of the UN steps before
      constexpr int UN = MTS == 2 ? 2 : 4, NB = MTS == 2 ? UN : UN / 2;
      uint32_t a[2][UN][4], b[2][NB][4];
      auto load = [&](int i0, uint32_t (&fa)[UN][4], uint32_t (&fb)[NB][4]) {
#pragma unroll
        for (int u = 0; u < UN; ++u) {
          const int i = min(i0 + u, steps - 1);
          ldmatrix_x4(qa + i * 32, fa[u][0], fa[u][1], fa[u][2], fa[u][3]);
          if (MTS == 2 || u % 2 == 0) {
            const int e = MTS == 2 ? i : i & ~1, f = MTS == 2 ? u : u / 2;
            ldmatrix_x4(ka + (e >> 2) * LA_BLOCK + ((((e & 3) * 2 + khi) ^ sw) << 4), fb[f][0],
                        fb[f][1], fb[f][2], fb[f][3]);
          }
        }
      };
      auto multiply = [&](int i0, uint32_t (&fa)[UN][4], uint32_t (&fb)[NB][4]) {
#pragma unroll
        for (int u = 0; u < UN; ++u)
          if (i0 + u < steps) {
            if (MTS == 2) {
              mma_bf16_16816(s[u & 1][0], fa[u], fb[u % NB][0], fb[u % NB][1]);
              mma_bf16_16816(s[u & 1][NK - 1], fa[u], fb[u % NB][2], fb[u % NB][3]);
            } else {
              mma_bf16_16816(s[u & 1][0], fa[u], fb[u / 2][(u & 1) * 2],
                             fb[u / 2][(u & 1) * 2 + 1]);
            }
          }
      };
      load(0, a[0], b[0]);
      for (int i0 = 0; i0 < steps; i0 += 2 * UN) {
        load(i0 + UN, a[1], b[1]);
        multiply(i0, a[0], b[0]);
        load(i0 + 2 * UN, a[0], b[0]);
        multiply(i0 + UN, a[1], b[1]);
      }
      float x[NK][4], t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
      for (int j = 0; j < NK; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = k0 + key0 + j * 8 + tq * 2 + e;
          x[j][e] = key < lim0 ? (s[0][j][e] + s[1][j][e]) * p.scale_log2 : -INFINITY;
          x[j][2 + e] = key < lim1 ? (s[0][j][2 + e] + s[1][j][2 + e]) * p.scale_log2 : -INFINITY;
          t0 = fmaxf(t0, x[j][e]);
          t1 = fmaxf(t1, x[j][2 + e]);
        }
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, o));
        t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, o));
      }
      if (tq == 0) {
        m_warp[warp * HT + row0] = t0;
        m_warp[warp * HT + row1] = t1;
      }
      named_bar_sync(1 + sub, 128);
      // the other warps of this tile that have these rows
#pragma unroll
      for (int w = 0; w < (MTS == 2 ? 2 : 4); ++w) {
        const float* mw = m_warp + (sub * 4 + (MTS == 2 ? w * 2 + mt : w)) * HT;
        t0 = fmaxf(t0, mw[row0]);
        t1 = fmaxf(t1, mw[row1]);
      }
      float p0 = -INFINITY, p1 = -INFINITY;
      if (n > 0) {
        ok = ok && mbar_wait(&m_full[sub ^ 1], (uint32_t)((n - 1) >> 1) & 1u, LA_WAIT_LIMIT);
        p0 = m_run[(sub ^ 1) * HT + row0];
        p1 = m_run[(sub ^ 1) * HT + row1];
        t0 = fmaxf(t0, p0);
        t1 = fmaxf(t1, p1);
      }
      const float z0 = t0 == -INFINITY ? 0.f : t0, z1 = t1 == -INFINITY ? 0.f : t1;
      const bool writes = tq == 0 && key0 == 0;
      if (writes) {
        m_run[sub * HT + row0] = t0;
        m_run[sub * HT + row1] = t1;
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&m_full[sub]);
      l0 *= fast_exp2(m0 - z0);
      l1 *= fast_exp2(m1 - z1);
      m0 = t0;
      m1 = t1;
#pragma unroll
      for (int j = 0; j < NK; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          x[j][e] = fast_exp2(x[j][e] - z0);
          x[j][2 + e] = fast_exp2(x[j][2 + e] - z1);
          l0 += x[j][e];
          l1 += x[j][2 + e];
        }
      if (n >= 2)
        ok = ok && mbar_wait(&p_empty[sub], (uint32_t)(n / 2 - 1) & 1u, LA_WAIT_LIMIT);
      uint16_t* ph = P + sub * 2 * HT * LA_PPITCH + key0 + tq * 2;
#pragma unroll
      for (int j = 0; j < NK; ++j) {
        uint32_t hi, lo;
        split_bf16(x[j][0], x[j][1], &hi, &lo);
        *reinterpret_cast<uint32_t*>(ph + row0 * LA_PPITCH + j * 8) = hi;
        *reinterpret_cast<uint32_t*>(ph + (HT + row0) * LA_PPITCH + j * 8) = lo;
        split_bf16(x[j][2], x[j][3], &hi, &lo);
        *reinterpret_cast<uint32_t*>(ph + row1 * LA_PPITCH + j * 8) = hi;
        *reinterpret_cast<uint32_t*>(ph + (HT + row1) * LA_PPITCH + j * 8) = lo;
      }
      if (writes) {
        alpha[sub * HT + row0] = p0 == -INFINITY ? 1.f : fast_exp2(p0 - z0);
        alpha[sub * HT + row1] = p1 == -INFINITY ? 1.f : fast_exp2(p1 - z1);
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[sub]);
    }
    if (!ok && p.status) atomicOr(p.status, FK_DEV_WAIT_TIMEOUT);
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      l0 += __shfl_xor_sync(0xffffffffu, l0, o);
      l1 += __shfl_xor_sync(0xffffffffu, l1, o);
    }
    // sums relative to the last maximum this warp has seen; rows it does not have stay out
    for (int r = lane; r < HT; r += 32) l_warp[warp * HT + r] = 0.f;
    __syncwarp();
    if (tq == 0) {
      l_warp[warp * HT + row0] = l0;
      l_warp[warp * HT + row1] = l1;
    }
    if (tiles < 2 && sub == 1 && v == 0)
      for (int r = lane; r < HT; r += 32) m_run[HT + r] = -INFINITY;
    if (tiles < 1 && sub == 0 && v == 0)
      for (int r = lane; r < HT; r += 32) m_run[r] = -INFINITY;
    named_bar_sync(4, LA_GROUP);
    if (tid < HT) {
      const float ma = m_run[tid], mb = m_run[HT + tid], mx = fmaxf(ma, mb);
      const float z = mx == -INFINITY ? 0.f : mx;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w)
        l += l_warp[w * HT + tid] * fast_exp2((w < 4 ? ma : mb) - z);
      inv_l[tid] = l > 0.f ? 1.0f / l : 0.f;
      if (p.splits > 1 && tid < n_rows)
        p.ml[(int64_t)split * p.flat_rows + first + tid] = make_float2(mx, l);
    }
    named_bar_sync(3, 2 * LA_GROUP);
    return;
  }

  // -------------------------------- values ---------------------------------
  float acc[MTS][RN][4];
#pragma unroll
  for (int a = 0; a < MTS; ++a)
#pragma unroll
    for (int j = 0; j < RN; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[a][j][i] = 0.f;
  const int col0 = (warp - LA_GROUP / 32) * RN * 8;
  for (int n = 0; n < tiles; ++n) {
    const int buf = n & 1, st = n % p.ring;
    ok = ok && mbar_wait(&full[st], (uint32_t)(n / p.ring) & 1u, LA_WAIT_LIMIT);
    ok = ok && mbar_wait(&p_full[buf], (uint32_t)(n >> 1) & 1u, LA_WAIT_LIMIT);
    const uint32_t tile = smem_u32(K + st * tile_bytes) + (lane & 15) * 128;
    const uint16_t* Ph = P + buf * 2 * HT * LA_PPITCH;
    const uint16_t* Pl = Ph + HT * LA_PPITCH;
    if (col0 < p.lo) {
#pragma unroll
      for (int a = 0; a < MTS; ++a) {
        const float a0 = alpha[buf * HT + a * 16 + gr], a1 = alpha[buf * HT + a * 16 + gr + 8];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int j = 0; j < RN; ++j) {
            acc[a][j][0] *= a0; acc[a][j][1] *= a0;
            acc[a][j][2] *= a1; acc[a][j][3] *= a1;
          }
        }
      }
#pragma unroll
      for (int kt = 0; kt < LA_KEYS / 16; ++kt) {
        uint32_t ph[MTS][4], pl[MTS][4];
#pragma unroll
        for (int a = 0; a < MTS; ++a) {
          const uint32_t off = (a * 16 + (lane & 15)) * LA_PPITCH + kt * 16 + (lane >> 4) * 8;
          ldmatrix_x4(smem_u32(Ph + off), ph[a][0], ph[a][1], ph[a][2], ph[a][3]);
          ldmatrix_x4(smem_u32(Pl + off), pl[a][0], pl[a][1], pl[a][2], pl[a][3]);
        }
        constexpr int GRP = RN / 2 < 4 / MTS ? RN / 2 : 4 / MTS;   // 16-column groups at a time
#pragma unroll
        for (int j0 = 0; j0 < RN / 2; j0 += GRP) {
          uint32_t b[GRP][4];
#pragma unroll
          for (int j = 0; j < GRP; ++j) {
            // columns beyond the latent are not stored: any column of the row will do
            const int c = min(col0 + (j0 + j) * 16, p.lo - 16);
            ldmatrix_x4_trans(tile + kt * 16 * 128 + (c >> 6) * LA_BLOCK +
                                  ((((c >> 3) & 7) + (lane >> 4)) ^ sw) * 16,
                              b[j][0], b[j][1], b[j][2], b[j][3]);
          }
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int a = 0; a < MTS; ++a)
#pragma unroll
              for (int j = 0; j < GRP; ++j) {
                mma_bf16_16816(acc[a][2 * (j0 + j)], part ? pl[a] : ph[a], b[j][0], b[j][1]);
                mma_bf16_16816(acc[a][2 * (j0 + j) + 1], part ? pl[a] : ph[a], b[j][2], b[j][3]);
              }
        }
      }
    }
    __syncwarp();
    if (lane == 0) {
      mbar_arrive(&empty[st]);
      mbar_arrive(&p_empty[buf]);
    }
  }
  named_bar_sync(3, 2 * LA_GROUP);
  if (p.splits > 1 && tiles == 0) return;
#pragma unroll
  for (int a = 0; a < MTS; ++a)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = a * 16 + gr + e * 8;
      if (r >= n_rows) continue;
      if (p.splits > 1) {
        float* o = p.part + ((int64_t)split * p.flat_rows + first + r) * p.lo;
#pragma unroll
        for (int j = 0; j < RN; ++j) {
          const int c = col0 + j * 8 + tq * 2;
          if (c < p.lo)
            *reinterpret_cast<float2*>(o + c) = make_float2(acc[a][j][e * 2], acc[a][j][e * 2 + 1]);
        }
      } else {
        const float inv = inv_l[r];
        uint16_t* o = p.out + (first + r) * p.out_pitch;
#pragma unroll
        for (int j = 0; j < RN; ++j) {
          const int c = col0 + j * 8 + tq * 2;
          if (c < p.lo)
            *reinterpret_cast<uint32_t*>(o + c) =
                pack_bf16(acc[a][j][e * 2] * inv, acc[a][j][e * 2 + 1] * inv);
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

// [rows, channels] bf16 pool: box = 64 channels x `run` rows, 128B swizzle
static int la_map(const void* ptr, int64_t rows, int64_t cols, int run, CUtensorMap* out) {
  struct Entry { const void* ptr; int64_t rows, cols; int run; CUtensorMap map; };
  static std::mutex mu;
  static std::vector<Entry> maps;
  std::lock_guard<std::mutex> lk(mu);
  for (const Entry& e : maps)
    if (e.ptr == ptr && e.rows == rows && e.cols == cols && e.run == run) {
      *out = e.map;
      return FK_OK;
    }
  tensormap_encode_fn enc = get_tensormap_encode();
  FK_REQUIRE(enc != nullptr, FK_ERR_CUDA,
             "cuTensorMapEncodeTiled not available from the driver");
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
  cuuint32_t box[2] = {64, (cuuint32_t)run};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims,
                   strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  FK_REQUIRE(r == CUDA_SUCCESS, FK_ERR_CUDA, "cuTensorMapEncodeTiled failed with code %d",
             (int)r);
  if (maps.size() > 1024) maps.clear();
  maps.push_back({ptr, rows, cols, run, *out});
  return FK_OK;
}

template <int HT, int RN>
static int launch_latent(LatentAttnParams& p, dim3 grid, cudaStream_t s) {
  p.ring = la_ring(HT, p.lk);
  FK_REQUIRE(p.ring > 0, FK_ERR_UNSUPPORTED, "fk_latent_attn: rows of %d elements", p.lk);
  const int smem = la_smem(HT, p.lk, p.ring);
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, latent_attn_kernel<HT, RN>, 232448));
  p.run = LA_KEYS;                       // keys that surely lie in one page
  while (p.block_size % p.run) p.run /= 2;
  CUtensorMap map;
  const int rc = la_map(p.cache, (int64_t)p.num_blocks * p.block_size, p.cache_pitch, p.run, &map);
  if (rc != FK_OK) return rc;
  FK_CUDA_OK(launch_kernel(latent_attn_kernel<HT, RN>, grid, dim3(LA_THREADS), (size_t)smem, s,
                           map, p));
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

int fk_latent_attn_supported(int heads, int rank, int rot) {
  return heads > 0 && rank > 0 && rank <= 512 && rot >= 0 &&
         la_ring(heads <= 16 ? 16 : 32, (rank + rot + 15) / 16 * 16) > 0;
}

/* Key ranges a call with these sizes splits its rows into. */
int fk_latent_attn_splits(int num_seqs, int64_t max_q, int heads, int64_t max_keys) {
  const int ht = heads <= 16 ? 16 : 32;
  const int64_t tiles = (max_q * heads + ht - 1) / ht * num_seqs;
  if (tiles <= 0) return 1;
  int64_t s = (int64_t)sm_count() / tiles;
  const int64_t most = (max_keys + 127) / 128;
  s = s < most ? s : most;
  return (int)(s < 1 ? 1 : s > 32 ? 32 : s);
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
  FK_REQUIRE(fk_latent_attn_supported(heads, rank, rot), FK_ERR_UNSUPPORTED,
             "fk_latent_attn: rank %d with %d rotated channels", rank, rot);
  const int lk = (rank + rot + 15) / 16 * 16, lo = (rank + 15) / 16 * 16;
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
  const int ht = heads <= 16 ? 16 : 32;
  const int64_t tiles = (max_seqlen_q * heads + ht - 1) / ht;
  FK_REQUIRE(tiles <= 0x7fffffff && num_seqs <= 65535 && splits <= 65535 &&
                 p.flat_rows <= 0x7fffffff,
             FK_ERR_UNSUPPORTED, "fk_latent_attn: too many rows");
  const dim3 grid((unsigned)tiles, (unsigned)num_seqs, (unsigned)splits);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int rc;
  if (ht == 16)
    rc = rank <= 128 ? launch_latent<16, 2>(p, grid, s)
         : rank <= 256 ? launch_latent<16, 4>(p, grid, s) : launch_latent<16, 8>(p, grid, s);
  else
    rc = rank <= 128 ? launch_latent<32, 2>(p, grid, s)
         : rank <= 256 ? launch_latent<32, 4>(p, grid, s) : launch_latent<32, 8>(p, grid, s);
  if (rc != FK_OK || splits == 1) return rc;
  FK_CUDA_OK(launch_kernel(latent_merge_kernel, dim3((unsigned)p.flat_rows), dim3(128), 0, s, p));
  count_launch();
  return FK_OK;
}

}  // extern "C"
