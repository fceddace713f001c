// Kernels without shape restrictions, for the number format and the head sizes the
// tensor-core kernels do not take:
//
//   fk_gemm_f32         y = x w^T (+ bias) in true fp32 (no tensor cores, so no reduced
//                       precision), any m, n
//   fk_paged_attn_any   causal attention over the paged NHD pool, bf16 or fp32, any
//                       head size up to 1152 and any query / KV head ratio; prompt
//                       portions and single decoded tokens alike
#include "fk_types.cuh"

#include <cmath>

namespace fk {

constexpr int GF_M = 64, GF_N = 64, GF_K = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(
    const float* __restrict__ x, int64_t x_stride, const float* __restrict__ w,
    const float* __restrict__ bias, float* __restrict__ y, int64_t y_stride, int m, int n,
    int k) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float xs[GF_K][GF_M + 4], ws[GF_K][GF_N + 4];
  const int n0 = blockIdx.x * GF_N, m0 = blockIdx.y * GF_M;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;   // 64 rows x 4 float4
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += GF_K) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (k0 + lc < k) {      // k is a multiple of 4
      if (m0 + lr < m)
        a = *reinterpret_cast<const float4*>(x + (int64_t)(m0 + lr) * x_stride + k0 + lc);
      if (n0 + lr < n)
        b = *reinterpret_cast<const float4*>(w + (int64_t)(n0 + lr) * k + k0 + lc);
    }
    __syncthreads();
    xs[lc][lr] = a.x; xs[lc + 1][lr] = a.y; xs[lc + 2][lr] = a.z; xs[lc + 3][lr] = a.w;
    ws[lc][lr] = b.x; ws[lc + 1][lr] = b.y; ws[lc + 2][lr] = b.z; ws[lc + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < GF_K; ++kk) {
      const float4 av = *reinterpret_cast<const float4*>(&xs[kk][ty * 4]);
      const float4 bv = *reinterpret_cast<const float4*>(&ws[kk][tx * 4]);
      const float aa[4] = {av.x, av.y, av.z, av.w}, bb[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(aa[i], bb[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + ty * 4 + i;
    if (r >= m) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tx * 4 + j;
      if (c < n) y[(int64_t)r * y_stride + c] = acc[i][j] + (bias ? bias[c] : 0.f);
    }
  }
}

struct AnyAttnParams {
  const void* q; int64_t q_stride; void* out; int64_t out_stride;
  const void* k_cache; const void* v_cache;
  const int32_t* cu_q; const int32_t* kv_lens;
  const int32_t* block_tables; int64_t bt_stride;
  int num_seqs, hq, hkv, d, block_size, num_blocks;
  int64_t rows;
  float scale;
  int32_t* status;
};

constexpr int AA_WARPS = 4;

// One warp per (query row, head).  Lane j scores key k0 + j of each run of 32 keys;
// then the lanes own the value channels lane, lane + 32, ...
template <typename T, int CH>
__global__ void __launch_bounds__(AA_WARPS * 32) paged_attn_any_kernel(const AnyAttnParams p) {
  extern __shared__ float aa_q[];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* q = aa_q + warp * p.d;
  const int64_t items = p.rows * p.hq;
  for (int64_t it = (int64_t)blockIdx.x * AA_WARPS + warp; it < items;
       it += (int64_t)gridDim.x * AA_WARPS) {
    const int64_t row = it / p.hq;
    const int head = (int)(it - row * p.hq), kvh = head / (p.hq / p.hkv);
    int lo = 0, hi = p.num_seqs;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.cu_q[mid] <= row) lo = mid; else hi = mid;
    }
    const int q_len = p.cu_q[lo + 1] - p.cu_q[lo];
    int visible = p.kv_lens[lo] - q_len + (int)(row - p.cu_q[lo]) + 1;
    if (visible > p.kv_lens[lo]) visible = p.kv_lens[lo];
    __syncwarp();
    const T* qr = static_cast<const T*>(p.q) + row * p.q_stride + (int64_t)head * p.d;
    for (int c = lane; c < p.d; c += 32) q[c] = Elem<T>::load(qr + c) * p.scale;
    __syncwarp();
    const int32_t* bt = p.block_tables + (int64_t)lo * p.bt_stride;
    float acc[CH];
#pragma unroll
    for (int i = 0; i < CH; ++i) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int k0 = 0; k0 < visible; k0 += 32) {
      const int kk = k0 + lane;
      int64_t off = 0;
      float s = -INFINITY;
      if (kk < visible) {
        int page = bt[kk / p.block_size];
        if (page < 0 || page >= p.num_blocks) {
          if (p.status) atomicOr(p.status, FK_DEV_BAD_PAGE);
        } else {
          off = (((int64_t)page * p.block_size + kk % p.block_size) * p.hkv + kvh) * p.d;
          const T* kr = static_cast<const T*>(p.k_cache) + off;
          float s4[4] = {0.f, 0.f, 0.f, 0.f};
          for (int c = 0; c < p.d; c += 4) {
            const float4 kv = Elem<T>::load4(kr + c);
            s4[0] = fmaf(kv.x, q[c], s4[0]);
            s4[1] = fmaf(kv.y, q[c + 1], s4[1]);
            s4[2] = fmaf(kv.z, q[c + 2], s4[2]);
            s4[3] = fmaf(kv.w, q[c + 3], s4[3]);
          }
          s = (s4[0] + s4[1]) + (s4[2] + s4[3]);
        }
      }
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_new = fmaxf(m, mx);
      if (m_new == -INFINITY) continue;
      const float alpha = expf(m - m_new);
      m = m_new;
      const float pr = expf(s - m_new);
      l = l * alpha + warp_sum(pr);
#pragma unroll
      for (int i = 0; i < CH; ++i) acc[i] *= alpha;
      const int cnt = min(32, visible - k0);
      for (int j = 0; j < cnt; ++j) {
        const float pj = __shfl_sync(0xffffffffu, pr, j);
        const int64_t oj = __shfl_sync(0xffffffffu, off, j);
        const T* vr = static_cast<const T*>(p.v_cache) + oj;
#pragma unroll
        for (int i = 0; i < CH; ++i) {
          const int c = lane + i * 32;
          if (c < p.d) acc[i] = fmaf(pj, Elem<T>::load(vr + c), acc[i]);
        }
      }
    }
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    T* o = static_cast<T*>(p.out) + row * p.out_stride + (int64_t)head * p.d;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const int c = lane + i * 32;
      if (c < p.d) Elem<T>::store(o + c, acc[i] * inv);
    }
  }
}

template <typename T>
static cudaError_t launch_any(const AnyAttnParams& p, int grid, cudaStream_t s) {
  const size_t smem = (size_t)AA_WARPS * p.d * sizeof(float);
  if (p.d <= 64)
    return launch_kernel(paged_attn_any_kernel<T, 2>, dim3(grid), dim3(AA_WARPS * 32), smem, s, p);
  if (p.d <= 128)
    return launch_kernel(paged_attn_any_kernel<T, 4>, dim3(grid), dim3(AA_WARPS * 32), smem, s, p);
  if (p.d <= 512)
    return launch_kernel(paged_attn_any_kernel<T, 16>, dim3(grid), dim3(AA_WARPS * 32), smem, s, p);
  return launch_kernel(paged_attn_any_kernel<T, 36>, dim3(grid), dim3(AA_WARPS * 32), smem, s, p);
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_gemm_f32(const float* x, int64_t x_stride, const float* w, const float* bias, float* y,
                int64_t y_stride, int64_t m, int64_t n, int64_t k, fk_stream_t stream) {
  FK_REQUIRE(m >= 0 && n >= 0 && k > 0, FK_ERR_INVALID_ARG, "fk_gemm_f32: bad sizes");
  if (m == 0 || n == 0) return FK_OK;
  FK_REQUIRE(x && w && y, FK_ERR_INVALID_ARG, "fk_gemm_f32: null pointer");
  FK_REQUIRE(x_stride >= k && y_stride >= n, FK_ERR_INVALID_ARG,
             "fk_gemm_f32: row stride smaller than the row");
  FK_REQUIRE(k % 4 == 0 && x_stride % 4 == 0 && aligned16(x) && aligned16(w), FK_ERR_ALIGNMENT,
             "fk_gemm_f32: x and w need 16-byte aligned rows");
  FK_REQUIRE(n < (1ll << 31) && k < (1ll << 31) && (m + GF_M - 1) / GF_M <= 65535,
             FK_ERR_UNSUPPORTED, "fk_gemm_f32: dimension too large");
  const dim3 grid((unsigned)((n + GF_N - 1) / GF_N), (unsigned)((m + GF_M - 1) / GF_M));
  FK_CUDA_OK(launch_kernel(gemm_f32_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream),
                           x, x_stride, w, bias, y, y_stride, (int)m, (int)n, (int)k));
  count_launch();
  return FK_OK;
}

int fk_paged_attn_any(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                      const void* k_cache, const void* v_cache, int is_f32, int64_t num_blocks,
                      int block_size, const int32_t* cu_seqlens_q, const int32_t* kv_lens,
                      const int32_t* block_tables, int64_t block_table_stride, int num_seqs,
                      int64_t rows, int num_q_heads, int num_kv_heads, int head_dim,
                      float softmax_scale, int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && num_seqs >= 0 && head_dim > 0 && num_q_heads > 0 && num_kv_heads > 0,
             FK_ERR_INVALID_ARG, "fk_paged_attn_any: bad sizes");
  if (rows == 0 || num_seqs == 0) return FK_OK;
  FK_REQUIRE(q && out && k_cache && v_cache && cu_seqlens_q && kv_lens && block_tables,
             FK_ERR_INVALID_ARG, "fk_paged_attn_any: null pointer");
  FK_REQUIRE(num_q_heads % num_kv_heads == 0 && block_size > 0 && num_blocks > 0 &&
                 num_blocks < (1ll << 31) && block_table_stride > 0,
             FK_ERR_INVALID_ARG, "fk_paged_attn_any: bad sizes");
  FK_REQUIRE(head_dim % 4 == 0 && head_dim <= 1152, FK_ERR_UNSUPPORTED,
             "fk_paged_attn_any: head_dim %d must be a multiple of 4, at most 1152", head_dim);
  FK_REQUIRE(aligned16(k_cache) && aligned16(v_cache), FK_ERR_ALIGNMENT,
             "fk_paged_attn_any: caches must be 16-byte aligned");
  FK_REQUIRE(q_stride >= (int64_t)num_q_heads * head_dim &&
                 out_stride >= (int64_t)num_q_heads * head_dim,
             FK_ERR_INVALID_ARG, "fk_paged_attn_any: token stride too small");
  AnyAttnParams p{};
  p.q = q; p.q_stride = q_stride; p.out = out; p.out_stride = out_stride; p.k_cache = k_cache;
  p.v_cache = v_cache; p.cu_q = cu_seqlens_q; p.kv_lens = kv_lens; p.block_tables = block_tables;
  p.bt_stride = block_table_stride; p.num_seqs = num_seqs; p.hq = num_q_heads;
  p.hkv = num_kv_heads; p.d = head_dim; p.block_size = block_size; p.num_blocks = (int)num_blocks;
  p.rows = rows; p.scale = softmax_scale; p.status = status;
  const int64_t want = (rows * num_q_heads + AA_WARPS - 1) / AA_WARPS;
  const int64_t cap = (int64_t)sm_count() * 32;
  const int grid = (int)(want < cap ? want : cap);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32 ? launch_any<float>(p, grid, s) : launch_any<uint16_t>(p, grid, s));
  count_launch();
  return FK_OK;
}

}  // extern "C"
