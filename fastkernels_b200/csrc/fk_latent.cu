// Latent attention: one cached row per token, [latent (rank) | rotated key (rot)], shared by
// all heads.  With the key and value projections of a head taken into its query and its
// output ("absorbed"), a head's query is [W_uk^T q | rotated q], its keys are the cached rows
// and its values the first `rank` channels of them.
//
//   latent_prepare_kernel   norm of the latent, rotation of the shared key, store; rotation
//                           (and copy) of the queries
//   latent_gather_kernel    cached rows of a batch's sequences side by side
//   latent_attn_kernel      absorbed attention, bf16: portions and single tokens alike.  A
//                           CTA owns HT (token, head) rows of one sequence and a range of
//                           keys; key tiles of 64 rows are double-buffered and serve as K
//                           and as V
//   latent_merge_kernel     key ranges of a row -> one result
//
// Scores, softmax weights and sums are fp32; the weights enter the tensor product with the
// values as two bf16 parts.
#include "fk_types.cuh"

#include <cmath>

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
  int heads, lk, lo, block_size, num_blocks, splits;
  float scale_log2;
  int32_t* status;
};

constexpr int LA_THREADS = 256, LA_KEYS = 64;
constexpr int LA_SPITCH = LA_KEYS + 4, LA_PPITCH = LA_KEYS + 8;

__host__ __device__ constexpr int la_smem(int ht, int lk) {
  return (ht + 2 * LA_KEYS) * (lk + 8) * 2 + 32 * LA_SPITCH * 4 + 2 * ht * LA_PPITCH * 2 +
         ht * 4;
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src)
               : "memory");
}

template <int HT, int RN>
__global__ void __launch_bounds__(LA_THREADS, 1) latent_attn_kernel(const LatentAttnParams p) {
  extern __shared__ __align__(16) uint8_t la_raw[];
  pdl_launch_dependents();
  pdl_wait();
  constexpr int MTS = HT / 16;
  const int seq = blockIdx.y, split = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gr = lane >> 2, tq = lane & 3;
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

  const int kp = p.lk + 8;
  uint16_t* Q = reinterpret_cast<uint16_t*>(la_raw);
  uint16_t* K = Q + HT * kp;                              // two tiles
  float* S = reinterpret_cast<float*>(K + 2 * LA_KEYS * kp);       // [32][LA_SPITCH]
  uint16_t* Ph = reinterpret_cast<uint16_t*>(S + 32 * LA_SPITCH);
  uint16_t* Pl = Ph + HT * LA_PPITCH;
  float* alpha = reinterpret_cast<float*>(Pl + HT * LA_PPITCH);

  const int packs = p.lk >> 3;
  const int32_t* bt = p.block_tables + seq * p.bt_stride;
  auto load_tile = [&](int k0, uint16_t* dst) {
    for (int r = warp; r < LA_KEYS; r += LA_THREADS / 32) {
      const int key = k0 + r;
      const uint16_t* src = nullptr;
      if (key < k_end) {
        const int page = bt[key / p.block_size];
        if (page >= 0 && page < p.num_blocks)
          src = p.cache + ((int64_t)page * p.block_size + key % p.block_size) * p.cache_pitch;
        else if (lane == 0 && p.status)
          atomicOr(p.status, FK_DEV_BAD_PAGE);
      }
      for (int c = lane; c < packs; c += 32) {
        if (src) cp_async16(dst + r * kp + c * 8, src + c * 8);
        else *reinterpret_cast<uint4*>(dst + r * kp + c * 8) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  for (int i = tid; i < HT * packs; i += LA_THREADS) {
    const int r = i / packs, c = (i - r * packs) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < n_rows) v = *reinterpret_cast<const uint4*>(p.q + (first + r) * p.q_pitch + c);
    *reinterpret_cast<uint4*>(Q + r * kp + c) = v;
  }
  if (k_begin < k_end) load_tile(k_begin, K);

  // softmax: TPR threads per row, KPT keys each
  constexpr int TPR = LA_THREADS / HT, KPT = LA_KEYS / TPR;
  const int srow = tid / TPR, skey = (tid % TPR) * KPT;
  const int my_lim = srow < n_rows ? min(kv_len, before + (tok0 + srow) / p.heads) : 0;
  float m = -INFINITY, l = 0.f;

  float acc[MTS][RN][4];
#pragma unroll
  for (int a = 0; a < MTS; ++a)
#pragma unroll
    for (int j = 0; j < RN; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[a][j][i] = 0.f;
  const int col0 = warp * RN * 8;
  const int steps = p.lk >> 4;

  int stage = 0;
  for (int k0 = k_begin; k0 < k_end; k0 += LA_KEYS, stage ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const uint16_t* Kt = K + stage * LA_KEYS * kp;
    if (k0 + LA_KEYS < k_end) load_tile(k0 + LA_KEYS, K + (stage ^ 1) * LA_KEYS * kp);
    {
      // HT = 32: warps 0-3 rows 0-15, 4-7 rows 16-31.  HT = 16: each half of the channels.
      const int kg = (warp & 3) * 16, part = warp >> 2;
      const int mrow = MTS == 2 ? part * 16 : 0;
      const int s0 = MTS == 2 ? 0 : part * ((steps + 1) >> 1);
      const int s1 = MTS == 2 ? steps : part ? steps : (steps + 1) >> 1;
      float s[2][4] = {};
      const uint32_t qa = smem_u32(Q + (mrow + (lane & 15)) * kp + (lane >> 4) * 8);
      const uint32_t ka = smem_u32(Kt + (kg + (lane & 7) + (lane >> 4) * 8) * kp +
                                   ((lane >> 3) & 1) * 8);
#pragma unroll 4
      for (int i = s0; i < s1; ++i) {
        uint32_t a[4], b[4];
        ldmatrix_x4(qa + i * 32, a[0], a[1], a[2], a[3]);
        ldmatrix_x4(ka + i * 32, b[0], b[1], b[2], b[3]);
        mma_bf16_16816(s[0], a, b[0], b[1]);
        mma_bf16_16816(s[1], a, b[2], b[3]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          *reinterpret_cast<float2*>(S + (part * 16 + gr + e * 8) * LA_SPITCH + kg + j * 8 +
                                     tq * 2) = make_float2(s[j][e * 2], s[j][e * 2 + 1]);
    }
    __syncthreads();
    {
      float x[KPT], mx = m;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        float v = S[srow * LA_SPITCH + skey + i];
        if (MTS == 1) v += S[(16 + srow) * LA_SPITCH + skey + i];
        x[i] = k0 + skey + i < my_lim && k0 + skey + i < k_end ? v * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, x[i]);
      }
#pragma unroll
      for (int o = TPR / 2; o > 0; o >>= 1)
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float al = mx == -INFINITY ? 1.f : exp2f(m - mx);
      m = mx;
      l *= al;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        x[i] = mx == -INFINITY ? 0.f : exp2f(x[i] - mx);
        l += x[i];
      }
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        uint32_t hi, lo;
        split_bf16(x[i], x[i + 1], &hi, &lo);
        *reinterpret_cast<uint32_t*>(Ph + srow * LA_PPITCH + skey + i) = hi;
        *reinterpret_cast<uint32_t*>(Pl + srow * LA_PPITCH + skey + i) = lo;
      }
      if (tid % TPR == 0) alpha[srow] = al;
    }
    __syncthreads();
#pragma unroll
    for (int a = 0; a < MTS; ++a) {
      const float a0 = alpha[a * 16 + gr], a1 = alpha[a * 16 + gr + 8];
#pragma unroll
      for (int j = 0; j < RN; ++j) {
        acc[a][j][0] *= a0; acc[a][j][1] *= a0;
        acc[a][j][2] *= a1; acc[a][j][3] *= a1;
      }
    }
    if (col0 < p.lo) {
#pragma unroll
      for (int kt = 0; kt < LA_KEYS / 16; ++kt) {
        uint32_t ph[MTS][4], pl[MTS][4];
#pragma unroll
        for (int a = 0; a < MTS; ++a) {
          const uint32_t off = (a * 16 + (lane & 15)) * LA_PPITCH + kt * 16 + (lane >> 4) * 8;
          ldmatrix_x4(smem_u32(Ph + off), ph[a][0], ph[a][1], ph[a][2], ph[a][3]);
          ldmatrix_x4(smem_u32(Pl + off), pl[a][0], pl[a][1], pl[a][2], pl[a][3]);
        }
#pragma unroll
        for (int j = 0; j < RN; j += 2) {
          const int c = col0 + j * 8;
          if (c >= p.lo) break;
          uint32_t b[4];
          ldmatrix_x4_trans(smem_u32(Kt + (kt * 16 + (lane & 15)) * kp + c + (lane >> 4) * 8),
                            b[0], b[1], b[2], b[3]);
#pragma unroll
          for (int a = 0; a < MTS; ++a) {
            mma_bf16_16816(acc[a][j], ph[a], b[0], b[1]);
            mma_bf16_16816(acc[a][j + 1], ph[a], b[2], b[3]);
            mma_bf16_16816(acc[a][j], pl[a], b[0], b[1]);
            mma_bf16_16816(acc[a][j + 1], pl[a], b[2], b[3]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int o = TPR / 2; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  __syncthreads();
  if (p.splits > 1) {
    if (tid % TPR == 0 && srow < n_rows)
      p.ml[(int64_t)split * p.flat_rows + first + srow] = make_float2(m, l);
    if (k_begin >= k_end) return;
  } else if (tid % TPR == 0) {
    alpha[srow] = l > 0.f ? 1.0f / l : 0.f;
  }
  __syncthreads();
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
        const float inv = alpha[r];
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

// One CTA per (token, head) row.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t r = blockIdx.x;
  float mx = -INFINITY;
  for (int s = 0; s < p.splits; ++s) {
    const float2 v = p.ml[(int64_t)s * p.flat_rows + r];
    if (v.y > 0.f) mx = fmaxf(mx, v.x);
  }
  float l = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    const float2 v = p.ml[(int64_t)s * p.flat_rows + r];
    if (v.y > 0.f) l += v.y * exp2f(v.x - mx);
  }
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  for (int c = threadIdx.x * 4; c < p.lo; c += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < p.splits; ++s) {
      const float2 v = p.ml[(int64_t)s * p.flat_rows + r];
      if (v.y > 0.f)
        a = a + *reinterpret_cast<const float4*>(
                    p.part + ((int64_t)s * p.flat_rows + r) * p.lo + c) *
                    (exp2f(v.x - mx) * inv);
    }
    Elem<uint16_t>::store4(p.out + r * p.out_pitch + c, a);
  }
}

template <int HT, int RN>
static int launch_latent(const LatentAttnParams& p, dim3 grid, cudaStream_t s) {
  const int smem = la_smem(HT, p.lk);
  FK_REQUIRE(smem <= 232448, FK_ERR_UNSUPPORTED, "fk_latent_attn: rows of %d elements", p.lk);
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, latent_attn_kernel<HT, RN>, 232448));
  FK_CUDA_OK(launch_kernel(latent_attn_kernel<HT, RN>, grid, dim3(LA_THREADS), (size_t)smem, s, p));
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

/* Key ranges a call with these sizes splits its rows into. */
int fk_latent_attn_splits(int num_seqs, int64_t max_q, int heads, int row_elements,
                          int64_t max_keys) {
  const int ht = heads <= 16 ? 16 : 32;
  const int64_t tiles = (max_q * heads + ht - 1) / ht * num_seqs;
  if (tiles <= 0) return 1;
  const int per_sm = 232448 / (la_smem(ht, (row_elements + 15) / 16 * 16) + 1024);
  int64_t s = (int64_t)sm_count() * (per_sm > 2 ? 2 : per_sm < 1 ? 1 : per_sm) / tiles;
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
  FK_REQUIRE(rows >= 0 && num_seqs >= 0 && heads > 0 && rank > 0 && rot >= 0 && splits >= 1,
             FK_ERR_INVALID_ARG, "fk_latent_attn: bad sizes");
  if (rows == 0 || num_seqs == 0 || max_seqlen_q <= 0) return FK_OK;
  FK_REQUIRE(q && cache && out && cu_seqlens_q && kv_lens && block_tables, FK_ERR_INVALID_ARG,
             "fk_latent_attn: null pointer");
  FK_REQUIRE(rank <= 512, FK_ERR_UNSUPPORTED, "fk_latent_attn: rank %d above 512", rank);
  const int lk = (rank + rot + 15) / 16 * 16, lo = (rank + 15) / 16 * 16;
  FK_REQUIRE(cache_pitch >= lk && q_pitch >= lk && out_pitch >= lo && block_size > 0 &&
                 num_blocks > 0 && num_blocks < (1ll << 31),
             FK_ERR_INVALID_ARG, "fk_latent_attn: rows shorter than latent and rotated key, "
             "rounded up to 16 elements");
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
