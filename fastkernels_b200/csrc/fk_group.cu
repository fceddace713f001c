// Grouped projections y = act(x w_g^T + bias), g = 0 .. groups - 1, in two forms:
//
//   column groups   every group takes all rows, its own columns of x and of y
//                   (x + g x_group, y + g y_group): per-head products, and with one
//                   group a plain projection with fp32 output
//   row groups      group g takes the rows offsets[g] .. offsets[g + 1] of y (x rows the
//                   same, or gather[row]): experts of a mixture
//
// act >= 0: w_g has 2 n rows [gate; up] and y = act(x gate^T) * (x up^T),
// each with its part of the bias.
// bf16 operands with fp32 accumulation and bf16 or fp32 results, or true fp32.
//
//   group_any_kernel     fp32 FMA, any sizes (fp32 operands)
//   group_skinny_kernel  few rows: streams the weights straight into mma.sync fragments.
//                        A product may take its k in any order as long as both operands
//                        do, so a lane's 16 contiguous bytes of a row serve as the k's of
//                        two instructions: no shared memory, no shuffles.
//   group_large_kernel   many rows: tcgen05, 128 rows x 256 weight rows, TMA-fed,
//                        accumulators double-buffered in tensor memory
#include "fk_tcgen05.cuh"
#include "fk_types.cuh"

#include <mutex>
#include <unordered_map>

namespace fk {

struct GroupParams {
  const void* x; int64_t x_stride, x_group;
  const void* w; int64_t w_rows;               // weight rows per group (n, or 2 n)
  const float* bias;                           // [w_rows] or null
  void* y; int64_t y_stride, y_group;
  const int32_t* offsets; const int32_t* gather;
  int64_t rows;                                // column groups: rows; row groups: all rows
  int64_t x_rows;                              // rows of x (bounds of gather)
  int groups, n, k, act;
  int32_t* status;
};

__device__ __forceinline__ float group_act(float g, int kind) {
  return kind == FK_ACT_SILU ? g * sigmoid_f32(g) : gelu_tanh_f32(g);
}

// Row range of a group inside y; empty or clamped when the offsets are not a partition.
__device__ __forceinline__ void group_range(const GroupParams& p, int g, int64_t* first,
                                            int64_t* count) {
  if (!p.offsets) { *first = 0; *count = p.rows; return; }
  int64_t a = p.offsets[g], b = p.offsets[g + 1];
  if (a < 0 || b < a || b > p.rows) {
    if (p.status && threadIdx.x == 0) atomicOr(p.status, FK_DEV_BAD_SLOT);
    a = b = 0;
  }
  *first = a;
  *count = b - a;
}
__device__ __forceinline__ int64_t group_x_row(const GroupParams& p, int64_t row) {
  if (!p.gather) return row;
  const int64_t r = p.gather[row];
  if (r < 0 || r >= p.x_rows) {
    if (p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
    return 0;
  }
  return r;
}

// ------------------------------------------------------------------------- any size
constexpr int GA_M = 64, GA_N = 64, GA_K = 16;

template <bool ACT>
__global__ void __launch_bounds__(256) group_any_kernel(const GroupParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int NB = ACT ? 2 : 1;
  __shared__ float xs[GA_K][GA_M + 4], ws[NB][GA_K][GA_N + 4];
  const int g = blockIdx.z;
  int64_t first, count;
  group_range(p, g, &first, &count);
  const int n0 = blockIdx.x * GA_N;
  const int64_t m0 = (int64_t)blockIdx.y * GA_M;
  if (m0 >= count) return;
  const float* x = static_cast<const float*>(p.x) + (p.offsets ? 0 : g * p.x_group);
  const float* w = static_cast<const float*>(p.w) + (int64_t)g * p.w_rows * p.k;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;
  const bool x_on = m0 + lr < count, w_on = n0 + lr < p.n;
  const float* xr = x + (x_on ? group_x_row(p, first + m0 + lr) : 0) * p.x_stride;
  float acc[NB][4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += GA_K) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b[NB];
#pragma unroll
    for (int e = 0; e < NB; ++e) b[e] = a;
    if (k0 + lc < p.k) {
      if (x_on) a = *reinterpret_cast<const float4*>(xr + k0 + lc);
#pragma unroll
      for (int e = 0; e < NB; ++e)
        if (w_on)
          b[e] = *reinterpret_cast<const float4*>(w + ((int64_t)e * p.n + n0 + lr) * p.k + k0 + lc);
    }
    __syncthreads();
    xs[lc][lr] = a.x; xs[lc + 1][lr] = a.y; xs[lc + 2][lr] = a.z; xs[lc + 3][lr] = a.w;
#pragma unroll
    for (int e = 0; e < NB; ++e) {
      ws[e][lc][lr] = b[e].x; ws[e][lc + 1][lr] = b[e].y;
      ws[e][lc + 2][lr] = b[e].z; ws[e][lc + 3][lr] = b[e].w;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < GA_K; ++kk) {
      const float4 av = *reinterpret_cast<const float4*>(&xs[kk][ty * 4]);
      const float aa[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
      for (int e = 0; e < NB; ++e) {
        const float4 bv = *reinterpret_cast<const float4*>(&ws[e][kk][tx * 4]);
        const float bb[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[e][i][j] = fmaf(aa[i], bb[j], acc[e][i][j]);
      }
    }
  }
  float* y = static_cast<float*>(p.y) + (p.offsets ? 0 : g * p.y_group);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int64_t r = m0 + ty * 4 + i;
    if (r >= count) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tx * 4 + j;
      if (c >= p.n) continue;
      float v = acc[0][i][j] + (p.bias ? p.bias[c] : 0.f);
      if (ACT) v = group_act(v, p.act) * (acc[NB - 1][i][j] + (p.bias ? p.bias[p.n + c] : 0.f));
      y[(first + r) * p.y_stride + c] = v;
    }
  }
}

// ------------------------------------------------------------------------- few rows
// A warp = 16 weight rows (of gate and of up with ACT) of one group, and every ks-th chunk
// of 32 k's; the CTA's warps are ks parts of k by 16-row tiles.  Rows go 8 NT at a time,
// blocks of them over grid.z.
template <int NT, bool ACT, typename OUT>
__global__ void __launch_bounds__(256) group_skinny_kernel(const GroupParams p, int ks) {
  extern __shared__ float gs_red[];            // [warps][TILES 16][8 NT + 1]
  pdl_launch_dependents();
  constexpr int TILES = ACT ? 2 : 1;
  constexpr int COLS = 8 * NT, PITCH = COLS + 1;
  const int g = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int gr = lane >> 2, tq = lane & 3;
  const int kpart = warp % ks, fs = warps / ks;
  const int n0 = blockIdx.x * (16 * fs);
  const uint16_t* w = static_cast<const uint16_t*>(p.w) + (int64_t)g * p.w_rows * p.k;
  const uint16_t* wr[TILES][2];
#pragma unroll
  for (int e = 0; e < TILES; ++e)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      int r = n0 + (warp / ks) * 16 + h * 8 + gr;
      if (r >= p.n) r = p.n - 1;               // computed, not stored
      wr[e][h] = w + ((int64_t)e * p.n + r) * p.k + tq * 8;
    }
  pdl_wait();
  int64_t first, count;
  group_range(p, g, &first, &count);
  const uint16_t* x = static_cast<const uint16_t*>(p.x) + (p.offsets ? 0 : g * p.x_group);
  const int chunks = (p.k + 31) >> 5;
  constexpr int kUnit = 16 / (int)sizeof(OUT);
  const bool vec = p.y_stride % kUnit == 0 && p.y_group % kUnit == 0;
  for (int64_t t0 = (int64_t)blockIdx.z * COLS; t0 < count; t0 += (int64_t)gridDim.z * COLS) {
    const uint16_t* xr[NT];
    bool on[NT];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int64_t t = t0 + j * 8 + gr;
      on[j] = t < count;
      xr[j] = x + (on[j] ? group_x_row(p, first + t) : 0) * p.x_stride + tq * 8;
    }
    float acc[TILES][NT][4];
#pragma unroll
    for (int e = 0; e < TILES; ++e)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[e][j][i] = 0.f;
    constexpr int UN = TILES * 2 + NT <= 6 ? 4 : TILES * 2 + NT <= 8 ? 2 : 1;
    for (int c0 = kpart; c0 < chunks; c0 += ks * UN) {
      uint4 a[UN][TILES][2], b[UN][NT];
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int c = c0 + u * ks;
        const bool in = c * 32 + tq * 8 < p.k;
#pragma unroll
        for (int e = 0; e < TILES; ++e)
#pragma unroll
          for (int h = 0; h < 2; ++h)
            a[u][e][h] = in ? __ldg(reinterpret_cast<const uint4*>(wr[e][h] + c * 32))
                            : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
        for (int j = 0; j < NT; ++j)
          b[u][j] = in && on[j] ? *reinterpret_cast<const uint4*>(xr[j] + c * 32)
                                : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int u = 0; u < UN; ++u)
#pragma unroll
        for (int e = 0; e < TILES; ++e) {
          const uint32_t lo[4] = {a[u][e][0].x, a[u][e][1].x, a[u][e][0].y, a[u][e][1].y};
          const uint32_t hi[4] = {a[u][e][0].z, a[u][e][1].z, a[u][e][0].w, a[u][e][1].w};
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            mma_bf16_16816(acc[e][j], lo, b[u][j].x, b[u][j].y);
            mma_bf16_16816(acc[e][j], hi, b[u][j].z, b[u][j].w);
          }
        }
    }
    __syncthreads();
    float* mine = gs_red + warp * (TILES * 16 * PITCH);
#pragma unroll
    for (int e = 0; e < TILES; ++e)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          mine[(e * 16 + gr + (i >> 1) * 8) * PITCH + j * 8 + tq * 2 + (i & 1)] = acc[e][j][i];
    __syncthreads();
    OUT* y = static_cast<OUT*>(p.y) + (p.offsets ? 0 : g * p.y_group);
    const int lg = 4 + (fs > 1) + (fs > 2), feats = 16 * fs;     // fs: 1, 2 or 4
    const int live = (int)min((int64_t)COLS, count - t0);
    // one output of row r, column t of this CTA's block
    auto value = [&](int r, int t) {
      const int c = n0 + r;
      const float* part = gs_red + (r >> 4) * ks * (TILES * 16 * PITCH) + (r & 15) * PITCH + t;
      float v = p.bias && c < p.n ? p.bias[c] : 0.f;
      float up = ACT && p.bias && c < p.n ? p.bias[p.n + c] : 0.f;
      for (int q = 0; q < ks; ++q) {
        v += part[q * (TILES * 16 * PITCH)];
        if (ACT) up += part[q * (TILES * 16 * PITCH) + 16 * PITCH];
      }
      return ACT ? group_act(v, p.act) * up : v;
    };
    // enough outputs for all threads: VEC features each, 16 bytes
    constexpr int VEC = 16 / (int)sizeof(OUT);
    const int step = vec && feats * live >= (int)blockDim.x * VEC ? VEC : 1;
    for (int i = threadIdx.x * step; i < feats * live; i += blockDim.x * step) {
      const int r = i & (feats - 1), t = i >> lg;
      const int c = n0 + r;
      if (c >= p.n) continue;
      OUT* dst = y + (first + t0 + t) * p.y_stride + c;
      if (step == 1) {
        Elem<OUT>::store(dst, value(r, t));
        continue;
      }
      float v[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = value(r + e, t);
      if (c + VEC <= p.n) {
        if (sizeof(OUT) == 2)
          *reinterpret_cast<uint4*>(dst) =
              make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]),
                         pack_bf16(v[VEC > 4 ? 4 : 0], v[VEC > 4 ? 5 : 1]),
                         pack_bf16(v[VEC > 4 ? 6 : 2], v[VEC > 4 ? 7 : 3]));
        else
          *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e)
          if (c + e < p.n) Elem<OUT>::store(dst + e, v[e]);
      }
    }
  }
}

// ------------------------------------------------------------------------ many rows
// BN weight rows a tile: 256, or 32 for narrow products, which have only 64 rows a tile (the
// instruction still multiplies 128; the others are not loaded and their results not kept).
constexpr int GG_BM = 128, GG_BK = 64;
constexpr int GG_A_BYTES = GG_BM * GG_BK * 2;
constexpr int GG_MAX_GROUPS = 1024;
constexpr int GG_THREADS = 192;
template <int BN>
struct GgCfg {
  static constexpr int kRows = BN == 256 ? 128 : 64;
  static constexpr int kBBytes = BN * GG_BK * 2;
  static constexpr int kStageBytes = GG_A_BYTES + kBBytes;
  static constexpr int kLoadBytes = kRows * GG_BK * 2 + kBBytes;
  static constexpr int kStages = BN == 256 ? 4 : 8;
  static constexpr int kOffTiles = kStages * kStageBytes;      // first tile of every group
  static constexpr int kOffBar = kOffTiles + (GG_MAX_GROUPS + 8) * 4;
  static constexpr int kOffOut = kOffBar + 256;       // 4 warps x 32 rows x 128 bytes
  static constexpr int kSmem = kOffOut + 4 * 4096 + 1024;
  static_assert(kSmem <= 232448, "shared memory budget");
};

__device__ __forceinline__ uint64_t gg_ns() {
  uint64_t t;
  asm volatile("mov.u64 %0, %globaltimer;" : "=l"(t));
  return t;
}
__device__ __forceinline__ bool gg_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag,
                                        int32_t* status) {
  if (mbar_try_wait(bar, parity)) return true;
  const uint64_t t0 = gg_ns();
  for (;;) {
    for (int i = 0; i < 128; ++i)
      if (mbar_try_wait(bar, parity)) return true;
    if (*abort_flag) return false;
    if (gg_ns() - t0 > 2000000000ull) {
      *abort_flag = 1;
      if (status) atomicOr(status, FK_DEV_WAIT_TIMEOUT);
      return false;
    }
  }
}
__device__ __forceinline__ bool gg_wait_warp(uint64_t* bar, uint32_t parity,
                                             volatile int* abort_flag, int32_t* status) {
  return __all_sync(0xffffffffu, gg_wait(bar, parity, abort_flag, status) ? 1 : 0) != 0;
}

struct GgTile {
  int g, nt;
  int64_t row0, rows_left;   // first row (of y and x), rows of the group from there on
};

// Tiles of a group lie together, rows fastest.
template <int ROWS>
__device__ __forceinline__ GgTile gg_tile(const GroupParams& p, const int* first_tile, int ti,
                                          int n_tiles) {
  int lo = 0, hi = p.groups;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (first_tile[mid] <= ti) lo = mid; else hi = mid;
  }
  const int in_g = ti - first_tile[lo];
  const int mts = (first_tile[lo + 1] - first_tile[lo]) / n_tiles;
  const int mt = in_g % mts;
  GgTile t;
  t.g = lo;
  t.nt = in_g / mts;
  int64_t a = 0, b = p.rows;
  if (p.offsets) { a = p.offsets[lo]; b = p.offsets[lo + 1]; }
  t.row0 = a + (int64_t)mt * ROWS;
  t.rows_left = b - t.row0;
  return t;
}

// Adds bias[from + c .. from + c + 3]; columns beyond n are not stored.
__device__ __forceinline__ void gg_add_bias(const GroupParams& p, int from, int c, float& a,
                                            float& b, float& d, float& e) {
  const float* q = p.bias + from + c;
  if (c + 4 <= p.n && (p.n & 3) == 0) {
    const float4 v = __ldg(reinterpret_cast<const float4*>(q));
    a += v.x; b += v.y; d += v.z; e += v.w;
  } else {
    if (c < p.n) a += q[0];
    if (c + 1 < p.n) b += q[1];
    if (c + 2 < p.n) d += q[2];
    if (c + 3 < p.n) e += q[3];
  }
}

template <int BN, bool ACT, typename OUT>
__global__ void __launch_bounds__(GG_THREADS, 1)
group_large_kernel(const __grid_constant__ CUtensorMap tmap_x,
                   const __grid_constant__ CUtensorMap tmap_w, const GroupParams p) {
  using Cfg = GgCfg<BN>;
  extern __shared__ uint8_t gg_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gg_raw) + 1023) &
                                             ~uintptr_t(1023));
  int* first_tile = reinterpret_cast<int*>(smem + Cfg::kOffTiles);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Cfg::kOffBar);
  uint64_t* full = bars;
  uint64_t* empty = bars + Cfg::kStages;
  uint64_t* acc_full = bars + 2 * Cfg::kStages;       // [2]
  uint64_t* acc_empty = acc_full + 2;              // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(acc_empty + 3);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int TN = ACT ? BN / 2 : BN;      // outputs per tile
  const int n_tiles = (p.n + TN - 1) / TN;
  const int kb_total = (p.k + GG_BK - 1) / GG_BK;

  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < Cfg::kStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(&acc_full[b], 1);
      mbar_init(&acc_empty[b], 4);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmap_x);
    tma_prefetch_desc(&tmap_w);
  }
  if (warp == 1) tmem_alloc(tmem_slot, 512);
  pdl_wait();
  // running tile count of the groups
  if (warp == 0) {
    int base = 0;
    for (int g0 = 0; g0 < p.groups; g0 += 32) {
      int64_t f = 0, c = 0;
      const int g = g0 + lane;
      if (g < p.groups) {
        if (p.offsets) {
          f = p.offsets[g];
          c = p.offsets[g + 1] - f;
          if (f < 0 || c < 0 || f + c > p.rows) {
            if (p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
            c = 0;
          }
        } else {
          c = p.rows;
        }
      }
      const int mine = (int)((c + Cfg::kRows - 1) / Cfg::kRows) * n_tiles;
      int run = mine;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      if (g < p.groups) first_tile[g] = base + run - mine;
      base += __shfl_sync(0xffffffffu, run, 31);
    }
    if (lane == 0) first_tile[p.groups] = base;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_got = *tmem_slot;
  if (tmem_got != 0) {        // all 512 columns: the allocation starts at column 0
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_TMEM_BASE);
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_got, 512);
    return;
  }
  const int total = first_tile[p.groups];

  if (warp == 0) {
    if (lane == 0) {
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int ti = blockIdx.x; ti < total && ok; ti += gridDim.x) {
        const GgTile t = gg_tile<Cfg::kRows>(p, first_tile, ti, n_tiles);
        const int xc = p.offsets ? 0 : (int)(t.g * p.x_group);
        const int wrow = (int)(t.g * p.w_rows) + t.nt * TN;
        for (int kb = 0; kb < kb_total; ++kb) {
          if (!gg_wait(&empty[stage], phase ^ 1, abort_flag, p.status)) { ok = false; break; }
          uint8_t* dst = smem + stage * Cfg::kStageBytes;
          mbar_arrive_expect_tx(&full[stage], (uint32_t)Cfg::kLoadBytes);
          tma_load_2d(dst, &tmap_x, &full[stage], xc + kb * GG_BK, (int)t.row0);
          if (ACT) {
            tma_load_2d(dst + GG_A_BYTES, &tmap_w, &full[stage], kb * GG_BK, wrow);
            tma_load_2d(dst + GG_A_BYTES + Cfg::kBBytes / 2, &tmap_w, &full[stage], kb * GG_BK,
                        wrow + p.n);
          } else {
            tma_load_2d(dst + GG_A_BYTES, &tmap_w, &full[stage], kb * GG_BK, wrow);
          }
          if (++stage == Cfg::kStages) { stage = 0; phase ^= 1; }
        }
      }
    }
  } else if (warp == 1) {
    constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) |
                               ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
    int stage = 0;
    uint32_t phase = 0, done = 0;
    bool ok = true;
    for (int ti = blockIdx.x; ti < total && ok; ti += gridDim.x) {
      const uint32_t buf = done & 1u, use = done >> 1;
      if (use > 0) ok = gg_wait_warp(&acc_empty[buf], (use - 1) & 1u, abort_flag, p.status);
      if (!ok) break;
      tc_fence_after();
      for (int kb = 0; kb < kb_total; ++kb) {
        ok = gg_wait_warp(&full[stage], phase, abort_flag, p.status);
        if (!ok) break;
        tc_fence_after();
        const uint32_t a = smem_u32(smem + stage * Cfg::kStageBytes);
        const uint32_t b = a + GG_A_BYTES;
#pragma unroll
        for (int kk = 0; kk < GG_BK / 16; ++kk)
          tc_mma_bf16_elect(buf * BN, smem_desc_sw128(a + kk * 32),
                            smem_desc_sw128(b + kk * 32), idesc, (kb > 0 || kk > 0) ? 1u : 0u);
        tc_commit_elect(&empty[stage]);
        if (++stage == Cfg::kStages) { stage = 0; phase ^= 1; }
      }
      if (!ok) break;
      tc_commit_elect(&acc_full[buf]);
      ++done;
    }
  } else {
    const int q = warp & 3;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    uint32_t done = 0;
    for (int ti = blockIdx.x; ti < total; ti += gridDim.x) {
      const GgTile t = gg_tile<Cfg::kRows>(p, first_tile, ti, n_tiles);
      const uint32_t buf = done & 1u, use = done >> 1;
      if (!gg_wait(&acc_full[buf], use & 1u, abort_flag, p.status)) break;
      tc_fence_after();
      // rows of this warp that exist
      const int rows = (int)max((int64_t)0, min((int64_t)32, min((int64_t)Cfg::kRows,
                                                                 t.rows_left) - q * 32));
      OUT* y = static_cast<OUT*>(p.y) + (p.offsets ? 0 : t.g * p.y_group) +
               (t.row0 + q * 32) * p.y_stride;
      const int n0 = t.nt * TN;
      // 128 bytes of every row at a time, through shared memory: a warp then stores whole
      // lines.  16-byte piece c of a row lies at c ^ (row & 7).
      constexpr int CH = 128 / (int)sizeof(OUT) < TN ? 128 / (int)sizeof(OUT) : TN;   // columns
      uint8_t* stage_out = smem + Cfg::kOffOut + q * 4096;
#pragma unroll 1
      for (int c0 = 0; c0 < TN; c0 += CH) {
        if (n0 + c0 >= p.n) break;
        __syncwarp();
#pragma unroll
        for (int c = 0; c < CH; c += 32) {
          uint32_t v[32], u[ACT ? 32 : 1];
          tc_ld32(lane_addr + buf * BN + c0 + c, v);
          if (ACT) tc_ld32(lane_addr + buf * BN + BN / 2 + c0 + c, u);
          tc_wait_ld();
          float f[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            f[i] = __uint_as_float(v[i]);
          }
          if (p.bias) {
#pragma unroll
            for (int i = 0; i < 32; i += 4)
              gg_add_bias(p, 0, n0 + c0 + c + i, f[i], f[i + 1], f[i + 2], f[i + 3]);
          }
          if (ACT) {
#pragma unroll
            for (int i = 0; i < 32; i += 4) {
              float up[4];
#pragma unroll
              for (int j = 0; j < 4; ++j) up[j] = __uint_as_float(u[ACT ? i + j : 0]);
              if (p.bias) gg_add_bias(p, p.n, n0 + c0 + c + i, up[0], up[1], up[2], up[3]);
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                const float g = f[i + j];
                f[i + j] = (p.act == FK_ACT_SILU
                                ? silu_f32(g) : __fdividef(g, 1.0f + __expf(-gelu_tanh_arg(g)))) *
                           up[j];
              }
            }
          }
          constexpr int PER = 16 / (int)sizeof(OUT);
#pragma unroll
          for (int i = 0; i < 32; i += PER) {
            uint4 w;
            if (sizeof(OUT) == 2)
              w = make_uint4(pack_bf16(f[i], f[i + 1]), pack_bf16(f[i + 2], f[i + 3]),
                             pack_bf16(f[i + 4 < 32 ? i + 4 : 0], f[i + 5 < 32 ? i + 5 : 0]),
                             pack_bf16(f[i + 6 < 32 ? i + 6 : 0], f[i + 7 < 32 ? i + 7 : 0]));
            else
              w = make_uint4(__float_as_uint(f[i]), __float_as_uint(f[i + 1]),
                             __float_as_uint(f[i + 2]), __float_as_uint(f[i + 3]));
            const int piece = (c + i) / PER;
            *reinterpret_cast<uint4*>(stage_out + lane * 128 + ((piece ^ (lane & 7)) << 4)) = w;
          }
        }
        __syncwarp();
        const int piece = lane & 7;
        const int col = n0 + c0 + piece * (16 / (int)sizeof(OUT));
#pragma unroll
        for (int r = lane >> 3; r < 32; r += 4) {
          if (r >= rows || col >= p.n) continue;
          const uint4 w = *reinterpret_cast<const uint4*>(stage_out + r * 128 +
                                                          ((piece ^ (r & 7)) << 4));
          OUT* dst = y + r * p.y_stride + col;
          if (col + 16 / (int)sizeof(OUT) <= p.n) {
            *reinterpret_cast<uint4*>(dst) = w;
          } else {
            const OUT* e = reinterpret_cast<const OUT*>(&w);
            for (int j = 0; j < 16 / (int)sizeof(OUT); ++j)
              if (col + j < p.n) dst[j] = e[j];
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&acc_empty[buf]);
      ++done;
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_got, 512);
  }
}

// ----------------------------------------------------------------------------- host
struct GgKey {
  const void* ptr; int64_t rows, cols, stride; int box_rows;
  bool operator==(const GgKey& o) const {
    return ptr == o.ptr && rows == o.rows && cols == o.cols && stride == o.stride &&
           box_rows == o.box_rows;
  }
};
struct GgHash {
  size_t operator()(const GgKey& k) const {
    return std::hash<const void*>()(k.ptr) ^
           std::hash<int64_t>()(k.rows * 1315423911ll + k.cols * 2654435761ll + k.stride +
                                k.box_rows * 7919ll);
  }
};
static std::mutex g_gg_mu;
static std::unordered_map<GgKey, CUtensorMap, GgHash> g_gg_maps;

// [rows, cols] bf16 with a row stride: box = 64 columns x box_rows rows, 128B swizzle
static int gg_map(const void* ptr, int64_t rows, int64_t cols, int64_t stride, int box_rows,
                  CUtensorMap* out) {
  GgKey key{ptr, rows, cols, stride, box_rows};
  std::lock_guard<std::mutex> lk(g_gg_mu);
  auto it = g_gg_maps.find(key);
  if (it != g_gg_maps.end()) {
    *out = it->second;
    return FK_OK;
  }
  tensormap_encode_fn enc = get_tensormap_encode();
  FK_REQUIRE(enc != nullptr, FK_ERR_CUDA,
             "cuTensorMapEncodeTiled not available from the driver");
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)stride * 2};
  cuuint32_t box[2] = {GG_BK, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1, 1};
  CUtensorMap m;
  CUresult r = enc(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims,
                   strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  FK_REQUIRE(r == CUDA_SUCCESS, FK_ERR_CUDA, "cuTensorMapEncodeTiled failed with code %d",
             (int)r);
  if (g_gg_maps.size() > 4096) g_gg_maps.clear();
  g_gg_maps.emplace(key, m);
  *out = m;
  return FK_OK;
}

template <int NT, bool ACT, typename OUT>
static int launch_skinny_one(const GroupParams& p, int ks, int fs, cudaStream_t s) {
  constexpr int kPerWarp = (ACT ? 2 : 1) * 16 * (8 * NT + 1) * 4;
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, group_skinny_kernel<NT, ACT, OUT>, 8 * kPerWarp));
  const int64_t blocks = p.offsets ? 1 : (p.rows + 8 * NT - 1) / (8 * NT);
  const dim3 grid((unsigned)((p.n + 16 * fs - 1) / (16 * fs)), (unsigned)p.groups,
                  (unsigned)(blocks < 65535 ? blocks : 65535));
  FK_CUDA_OK(launch_kernel(group_skinny_kernel<NT, ACT, OUT>, grid, dim3(32u * ks * fs),
                           (size_t)ks * fs * kPerWarp, s, p, ks));
  count_launch();
  return FK_OK;
}
template <bool ACT, typename OUT>
static int launch_skinny(const GroupParams& p, int64_t expect, cudaStream_t s) {
  const int chunks = (p.k + 31) / 32;
  const int ks = chunks >= 16 ? 8 : chunks >= 8 ? 4 : chunks >= 4 ? 2 : 1;
  const int fs = ks == 8 ? 1 : ks == 1 ? 4 : 8 / ks;
  // rows per CTA: as many as keep the machine busy (more rows read the weights once)
  int64_t nt = expect <= 8 ? 1 : expect <= 16 ? 2 : expect <= 32 ? 4 : 8;
  if (!p.offsets) {
    const int64_t tiles = (int64_t)((p.n + 16 * fs - 1) / (16 * fs)) * p.groups;
    while (nt > 1 && tiles * ((p.rows + 8 * nt - 1) / (8 * nt)) < sm_count()) nt /= 2;
  }
  if (nt == 1) return launch_skinny_one<1, ACT, OUT>(p, ks, fs, s);
  if (nt == 2) return launch_skinny_one<2, ACT, OUT>(p, ks, fs, s);
  if (nt == 4) return launch_skinny_one<4, ACT, OUT>(p, ks, fs, s);
  return launch_skinny_one<8, ACT, OUT>(p, ks, fs, s);
}
template <int BN, bool ACT, typename OUT>
static int launch_large_one(const GroupParams& p, int64_t x_cols, cudaStream_t s) {
  constexpr int TN = ACT ? BN / 2 : BN;
  const int64_t n_tiles = (p.n + TN - 1) / TN;
  constexpr int kRows = GgCfg<BN>::kRows;
  const int64_t bound = p.offsets ? ((p.rows + kRows - 1) / kRows + p.groups) * n_tiles
                                  : (p.rows + kRows - 1) / kRows * n_tiles * p.groups;
  FK_REQUIRE(bound <= 0x7fffffff && p.rows < (1ll << 31) && p.groups * p.w_rows < (1ll << 31),
             FK_ERR_UNSUPPORTED, "fk_group_gemm: too many tiles");
  CUtensorMap mx, mw;
  int rc = gg_map(p.x, p.x_rows, x_cols, p.x_stride, kRows, &mx);
  if (rc != FK_OK) return rc;
  rc = gg_map(p.w, p.groups * p.w_rows, p.k, p.k, TN, &mw);
  if (rc != FK_OK) return rc;
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, group_large_kernel<BN, ACT, OUT>, GgCfg<BN>::kSmem));
  const int ctas = (int)(bound < sm_count() ? bound : sm_count());
  FK_CUDA_OK(launch_kernel(group_large_kernel<BN, ACT, OUT>, dim3((unsigned)ctas), dim3(GG_THREADS),
                           (size_t)GgCfg<BN>::kSmem, s, mx, mw, p));
  count_launch();
  return FK_OK;
}

template <bool ACT, typename OUT>
static int launch_large(const GroupParams& p, int64_t x_cols, cudaStream_t s) {
  if constexpr (!ACT) {
    if (p.n <= 32) return launch_large_one<32, ACT, OUT>(p, x_cols, s);
  }
  return launch_large_one<256, ACT, OUT>(p, x_cols, s);
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_group_gemm(const void* x, int64_t x_stride, int64_t x_group, int64_t x_rows,
                  const void* w, const float* bias, void* y, int64_t y_stride, int64_t y_group,
                  int is_f32, int y_f32, const int32_t* offsets, const int32_t* gather,
                  int64_t rows, int64_t expect_rows, int groups, int64_t n, int64_t k, int act,
                  int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && groups > 0 && n >= 0 && k > 0 && x_rows >= 0, FK_ERR_INVALID_ARG,
             "fk_group_gemm: bad sizes");
  if (rows == 0 || n == 0) return FK_OK;
  FK_REQUIRE(x && w && y, FK_ERR_INVALID_ARG, "fk_group_gemm: null pointer");
  FK_REQUIRE(!gather || offsets, FK_ERR_INVALID_ARG,
             "fk_group_gemm: only row groups can be gathered");
  FK_REQUIRE(gather || x_rows >= rows, FK_ERR_INVALID_ARG, "fk_group_gemm: x has too few rows");
  FK_REQUIRE(act < 0 || act == FK_ACT_SILU || act == FK_ACT_GELU_TANH, FK_ERR_INVALID_ARG,
             "fk_group_gemm: unknown activation %d", act);
  const int64_t x_cols = offsets ? k : (groups - 1) * x_group + k;
  FK_REQUIRE(x_group >= 0 && y_group >= 0 && x_stride >= x_cols &&
                 y_stride >= (offsets ? n : (groups - 1) * y_group + n) &&
                 (offsets || groups == 1 || y_group >= n),
             FK_ERR_INVALID_ARG, "fk_group_gemm: row stride smaller than the row");
  FK_REQUIRE(n < (1ll << 30) && k < (1ll << 30) && groups <= 65535, FK_ERR_UNSUPPORTED,
             "fk_group_gemm: dimension too large");
  const int unit = is_f32 ? 4 : 8;
  FK_REQUIRE(k % unit == 0 && x_stride % unit == 0 && x_group % unit == 0 && aligned16(x) &&
                 aligned16(w) && aligned16(y) && aligned16(bias),
             FK_ERR_ALIGNMENT, "fk_group_gemm: x and w need 16-byte aligned rows");
  GroupParams p{};
  p.x = x; p.x_stride = x_stride; p.x_group = x_group; p.x_rows = x_rows; p.w = w;
  p.w_rows = act >= 0 ? 2 * n : n; p.bias = bias; p.y = y; p.y_stride = y_stride;
  p.y_group = y_group; p.offsets = offsets; p.gather = gather; p.rows = rows; p.groups = groups;
  p.n = (int)n; p.k = (int)k; p.act = act; p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (is_f32) {
    FK_REQUIRE(y_f32, FK_ERR_INVALID_ARG, "fk_group_gemm: fp32 operands give an fp32 result");
    const int64_t my = (rows + GA_M - 1) / GA_M;
    FK_REQUIRE(my <= 65535, FK_ERR_UNSUPPORTED, "fk_group_gemm: too many rows");
    const dim3 grid((unsigned)((n + GA_N - 1) / GA_N), (unsigned)my, (unsigned)groups);
    FK_CUDA_OK(act >= 0 ? launch_kernel(group_any_kernel<true>, grid, dim3(256), 0, s, p)
                        : launch_kernel(group_any_kernel<false>, grid, dim3(256), 0, s, p));
    count_launch();
    return FK_OK;
  }
  FK_REQUIRE(act < 0 || !y_f32, FK_ERR_UNSUPPORTED,
             "fk_group_gemm: an activation gives a bf16 result");
  // 16-byte stores of the large form
  const bool dense_y = y_stride % (y_f32 ? 4 : 8) == 0 && y_group % (y_f32 ? 4 : 8) == 0;
  const bool large = expect_rows > 64 && !gather && dense_y && groups <= GG_MAX_GROUPS;
  if (large) {
    if (act >= 0) return launch_large<true, uint16_t>(p, x_cols, s);
    return y_f32 ? launch_large<false, float>(p, x_cols, s)
                 : launch_large<false, uint16_t>(p, x_cols, s);
  }
  if (act >= 0) return launch_skinny<true, uint16_t>(p, expect_rows, s);
  return y_f32 ? launch_skinny<false, float>(p, expect_rows, s)
               : launch_skinny<false, uint16_t>(p, expect_rows, s);
}

}  // extern "C"
