// Routing of a mixture of experts:
//
//   fk_moe_route    from fp32 router logits [rows, experts]: the `top` largest experts of
//                   every row (lowest index on ties), their softmax weights, and the
//                   order of all (row, choice) pairs by expert: pair i of row t lies at
//                   place[t, i] of the expert-sorted list, whose entry r belongs to row
//                   source[r]; expert e owns entries offsets[e] .. offsets[e + 1]
//   fk_gather_rows  y[r] = x[source[r]]
//
// Few rows take one CTA; many rows count per block of rows, scan the counts, place.
// The order of an expert's entries among themselves carries no meaning.
#include "fk_types.cuh"

#include <cmath>

namespace fk {

constexpr int MR_MAX_EXPERTS = 1024;
constexpr int MR_BLOCK_ROWS = 64;

struct RouteParams {
  const float* z; int64_t z_stride;
  int32_t* chosen;      // [rows, top] expert
  float* share;         // [rows, top]
  int32_t* place;       // [rows, top]
  int32_t* source;      // [rows * top]
  int32_t* offsets;     // [experts + 1]
  int32_t* counts;      // [blocks, experts]
  int64_t rows; int experts, top, blocks;
};

// Unsigned numbers in the order of the logits, never 0; NaN counts as the smallest.
__device__ __forceinline__ uint32_t route_key(float z) {
  const uint32_t u = __float_as_uint(z);
  if (z != z) return 1u;
  return max(u >> 31 ? ~u : u | 0x80000000u, 1u);
}
__device__ __forceinline__ float route_logit(uint32_t key) {
  return __uint_as_float(key >> 31 ? key & 0x7fffffffu : ~key);
}

// One warp: choices and weights of row t; lane l holds the logits l, l + 32, ...
template <int EPL>
__device__ __forceinline__ void route_row(const RouteParams& p, int64_t t, int lane) {
  const float* z = p.z + t * p.z_stride;
  uint32_t key[EPL];
#pragma unroll
  for (int i = 0; i < EPL; ++i)
    key[i] = lane + i * 32 < p.experts ? route_key(z[lane + i * 32]) : 0u;
  uint32_t taken = 0;                              // bit i: v[i] is chosen already
  float first = 0.f, total = 0.f;
  for (int j = 0; j < p.top; ++j) {
    // largest free logit, then the lowest index that has it; unsigned keys in the order of
    // the logits, 0 = nothing free
    uint32_t best = 0u;
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (!((taken >> i) & 1u)) best = max(best, key[i]);
    const uint32_t top = __reduce_max_sync(0xffffffffu, best);
    uint32_t mine = 0xffffffffu;
#pragma unroll
    for (int i = EPL - 1; i >= 0; --i)
      if (!((taken >> i) & 1u) && key[i] == top) mine = lane + i * 32;
    const int at = (int)__reduce_min_sync(0xffffffffu, mine);
    const float chosen = route_logit(top);
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    if (j == 0) first = chosen;
    const float w = expf(chosen - first);
    total += w;
    if (lane == 0) {
      p.chosen[t * p.top + j] = at;
      p.share[t * p.top + j] = w;
    }
  }
  __syncwarp();
  const float inv = 1.0f / total;
  for (int j = lane; j < p.top; j += 32) p.share[t * p.top + j] *= inv;
}

// Exclusive scan of cnt[0 .. n) into out[0 .. n], one warp.
__device__ __forceinline__ void warp_scan(const int* cnt, int* cursor, int32_t* out, int n,
                                          int lane) {
  int base = 0;
  for (int e0 = 0; e0 < n; e0 += 32) {
    const int e = e0 + lane;
    const int mine = e < n ? cnt[e] : 0;
    int run = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += up;
    }
    if (e < n) {
      cursor[e] = base + run - mine;
      out[e] = base + run - mine;
    }
    base += __shfl_sync(0xffffffffu, run, 31);
  }
  if (lane == 0) out[n] = base;
}

// SINGLE: everything.  Otherwise choices, weights and the counts of the block's rows.
template <bool SINGLE, int EPL>
__global__ void __launch_bounds__(1024) moe_route_kernel(const RouteParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int cnt[MR_MAX_EXPERTS], cursor[SINGLE ? MR_MAX_EXPERTS : 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int64_t t0 = SINGLE ? 0 : (int64_t)blockIdx.x * MR_BLOCK_ROWS;
  const int64_t t1 = SINGLE ? p.rows : min(p.rows, t0 + MR_BLOCK_ROWS);
  for (int e = threadIdx.x; e < p.experts; e += blockDim.x) cnt[e] = 0;
  for (int64_t t = t0 + warp; t < t1; t += warps) route_row<EPL>(p, t, lane);
  __syncthreads();
  for (int64_t i = t0 * p.top + threadIdx.x; i < t1 * p.top; i += blockDim.x)
    atomicAdd(&cnt[p.chosen[i]], 1);
  __syncthreads();
  if (!SINGLE) {
    for (int e = threadIdx.x; e < p.experts; e += blockDim.x)
      p.counts[(int64_t)blockIdx.x * p.experts + e] = cnt[e];
    return;
  }
  if (warp == 0) warp_scan(cnt, cursor, p.offsets, p.experts, lane);
  __syncthreads();
  for (int64_t i = threadIdx.x; i < p.rows * p.top; i += blockDim.x) {
    const int at = atomicAdd(&cursor[p.chosen[i]], 1);
    p.place[i] = at;
    p.source[at] = (int32_t)(i / p.top);
  }
}

// counts[block][expert] -> first entry of the block's rows within the expert-sorted list
__global__ void __launch_bounds__(1024) moe_scan_kernel(const RouteParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int cnt[MR_MAX_EXPERTS], cursor[MR_MAX_EXPERTS];
  const int e = threadIdx.x;
  if (e < p.experts) {
    int run = 0;
    constexpr int UN = 16;
    for (int b0 = 0; b0 < p.blocks; b0 += UN) {
      int32_t* c = p.counts + (int64_t)b0 * p.experts + e;
      int mine[UN];
#pragma unroll
      for (int i = 0; i < UN; ++i) mine[i] = b0 + i < p.blocks ? c[(int64_t)i * p.experts] : 0;
#pragma unroll
      for (int i = 0; i < UN; ++i)
        if (b0 + i < p.blocks) {
          c[(int64_t)i * p.experts] = run;
          run += mine[i];
        }
    }
    cnt[e] = run;
  }
  __syncthreads();
  if (threadIdx.x < 32) warp_scan(cnt, cursor, p.offsets, p.experts, threadIdx.x);
}

__global__ void __launch_bounds__(256) moe_place_kernel(const RouteParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int cursor[MR_MAX_EXPERTS];
  for (int e = threadIdx.x; e < p.experts; e += blockDim.x)
    cursor[e] = p.offsets[e] + p.counts[(int64_t)blockIdx.x * p.experts + e];
  __syncthreads();
  const int64_t t0 = (int64_t)blockIdx.x * MR_BLOCK_ROWS;
  const int64_t t1 = min(p.rows, t0 + MR_BLOCK_ROWS);
  for (int64_t i = t0 * p.top + threadIdx.x; i < t1 * p.top; i += blockDim.x) {
    const int at = atomicAdd(&cursor[p.chosen[i]], 1);
    p.place[i] = at;
    p.source[at] = (int32_t)(i / p.top);
  }
}

__global__ void __launch_bounds__(256) gather_rows_kernel(
    const uint4* __restrict__ x, int64_t x_packs, int64_t x_rows, const int32_t* __restrict__ source,
    uint4* __restrict__ y, int64_t rows, int packs, int32_t* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = 256 / 32;
  const int lane = threadIdx.x & 31;
  for (int64_t r = (int64_t)blockIdx.x * per + (threadIdx.x >> 5); r < rows;
       r += (int64_t)gridDim.x * per) {
    const int64_t src = source[r];
    if (src < 0 || src >= x_rows) {
      if (lane == 0 && status) atomicOr(status, FK_DEV_BAD_SLOT);
      continue;
    }
    for (int c = lane; c < packs; c += 32) y[r * packs + c] = x[src * x_packs + c];
  }
}

template <bool SINGLE>
static cudaError_t launch_route(const RouteParams& p, int grid, int threads, cudaStream_t s) {
  if (p.experts <= 64)
    return launch_kernel(moe_route_kernel<SINGLE, 2>, dim3(grid), dim3(threads), 0, s, p);
  if (p.experts <= 256)
    return launch_kernel(moe_route_kernel<SINGLE, 8>, dim3(grid), dim3(threads), 0, s, p);
  return launch_kernel(moe_route_kernel<SINGLE, 32>, dim3(grid), dim3(threads), 0, s, p);
}

}  // namespace fk

using namespace fk;

extern "C" {

int64_t fk_moe_route_counts(int64_t rows, int experts, int top) {
  if (rows * top <= 2048) return 0;
  return (rows + MR_BLOCK_ROWS - 1) / MR_BLOCK_ROWS * experts;
}

int fk_moe_route(const float* z, int64_t z_stride, int32_t* chosen, float* share, int32_t* place,
                 int32_t* source, int32_t* offsets, int32_t* counts, int64_t rows, int experts,
                 int top, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && experts > 0 && top > 0 && top <= experts, FK_ERR_INVALID_ARG,
             "fk_moe_route: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(z && chosen && share && place && source && offsets, FK_ERR_INVALID_ARG,
             "fk_moe_route: null pointer");
  FK_REQUIRE(z_stride >= experts, FK_ERR_INVALID_ARG, "fk_moe_route: bad stride");
  FK_REQUIRE(experts <= MR_MAX_EXPERTS && rows * top < (1ll << 31), FK_ERR_UNSUPPORTED,
             "fk_moe_route: %d experts or too many rows", experts);
  RouteParams p{};
  p.z = z; p.z_stride = z_stride; p.chosen = chosen; p.share = share; p.place = place;
  p.source = source; p.offsets = offsets; p.counts = counts; p.rows = rows;
  p.experts = experts; p.top = top;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (fk_moe_route_counts(rows, experts, top) == 0) {
    const int threads = rows >= 32 ? 1024 : rows >= 8 ? 512 : 256;
    FK_CUDA_OK(launch_route<true>(p, 1, threads, s));
    count_launch();
    return FK_OK;
  }
  FK_REQUIRE(counts, FK_ERR_WORKSPACE, "fk_moe_route: this many rows need counts");
  p.blocks = (int)((rows + MR_BLOCK_ROWS - 1) / MR_BLOCK_ROWS);
  FK_CUDA_OK(launch_route<false>(p, p.blocks, 512, s));
  FK_CUDA_OK(launch_kernel(moe_scan_kernel, dim3(1), dim3(1024), 0, s, p));
  FK_CUDA_OK(launch_kernel(moe_place_kernel, dim3((unsigned)p.blocks), dim3(256), 0, s, p));
  count_launch(3);
  return FK_OK;
}

int fk_gather_rows(const void* x, int64_t x_stride_bytes, int64_t x_rows, const int32_t* source,
                   void* y, int64_t rows, int64_t row_bytes, int32_t* status,
                   fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && row_bytes > 0 && x_rows >= 0, FK_ERR_INVALID_ARG,
             "fk_gather_rows: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(x && source && y, FK_ERR_INVALID_ARG, "fk_gather_rows: null pointer");
  FK_REQUIRE(row_bytes % 16 == 0 && x_stride_bytes % 16 == 0 && x_stride_bytes >= row_bytes &&
                 aligned16(x) && aligned16(y),
             FK_ERR_ALIGNMENT, "fk_gather_rows: rows must be 16-byte aligned");
  FK_REQUIRE(row_bytes < (1ll << 31), FK_ERR_UNSUPPORTED, "fk_gather_rows: row too long");
  const int64_t want = (rows + 7) / 8, cap = (int64_t)sm_count() * 16;
  FK_CUDA_OK(launch_kernel(gather_rows_kernel, dim3((unsigned)(want < cap ? want : cap)),
                           dim3(256), 0, static_cast<cudaStream_t>(stream), (const uint4*)x,
                           x_stride_bytes / 16, x_rows, source, (uint4*)y, rows,
                           (int)(row_bytes / 16), status));
  count_launch();
  return FK_OK;
}

}  // extern "C"
