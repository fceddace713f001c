// Generalized delta rule with a decay per key channel (linear attention with a
// matrix state per head), fp32 throughout:
//
//   S_t = diag(w_t) S_{t-1} - (a_t * u_t) (u_t^T S_{t-1}) + k_t v_t^T,   o_t = S_t^T r_t
//
//   w_t = exp(-c sigmoid(W2 tanh(y1) + w0)),  a_t = sigmoid(y_a + b_a),
//   u_t = k_t / sqrt(sum k_t^2 + eps_u)       (per head)
//
// Three kernels:
//   delta_prepare_kernel   everything of a token that does not depend on the state:
//                          w, u, a * u, k, r, v as fp32, packed per (head, token) so
//                          that a run of tokens of one head is one contiguous block
//   delta_scan_kernel      the recurrence.  The columns of S (value channels) are
//                          independent, so a column lives in the registers of LANES
//                          threads (8 key channels each); a CTA owns some columns of
//                          one head of one sequence and streams the packed tokens
//                          through a ring of shared-memory stages (bulk copies).
//                          A single decoded token and a prompt portion are the same
//                          code; the state comes from and returns to HBM once.
//   delta_output_kernel    per-head RMS norm of o, weight, output gate.
//
// State layout [slot][head][value channel][key channel (padded)], so that the
// threads of a column read 16-byte pieces that are adjacent across lanes.
#include "fk_types.cuh"

#include <cmath>

namespace fk {

constexpr int DL_FIELDS = 6;      // w, u, a * u, k, r, v
constexpr int DL_CPL = 8;         // key channels per thread
constexpr int DL_THREADS = 128;
constexpr int DL_STAGES = 3;
constexpr int DL_PREP_TOK = 16;   // tokens per CTA of the prepare kernel
constexpr int DL_MAX_DIM = 256;
constexpr uint32_t DL_WAIT_LIMIT = 1u << 20;

struct DeltaPrepParams {
  const void* r; const void* k; const void* v; const void* a; const void* y1;
  int64_t in_stride;                    // packed projection rows
  const void* w2; int64_t w2_stride;    // [heads * d, rank]
  const float* w0; const float* a_bias; // [heads * d]
  float* packed;                        // [heads][rows][DL_FIELDS][dp]
  int64_t rows; int heads, d, dp, rank;
  float decay_scale, unit_eps;
};

// CTA = 16 tokens of one head, thread = key channel.
template <typename T>
__global__ void __launch_bounds__(DL_MAX_DIM) delta_prepare_kernel(const DeltaPrepParams p) {
  extern __shared__ float dl_prep_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int rank_p = (p.rank + 3) & ~3;
  float* th = dl_prep_smem;                                 // [TOK][rank_p]
  float* ksq = th + DL_PREP_TOK * rank_p;                   // [warps][TOK]
  const int h = blockIdx.y;
  const int64_t t0 = (int64_t)blockIdx.x * DL_PREP_TOK;
  const int nt = (int)min((int64_t)DL_PREP_TOK, p.rows - t0);
  const int c = threadIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  for (int i = threadIdx.x; i < DL_PREP_TOK * rank_p; i += blockDim.x) {
    const int t = i / rank_p, r = i - t * rank_p;
    float z = 0.f;
    if (t < nt && r < p.rank)
      z = tanhf(Elem<T>::load(static_cast<const T*>(p.y1) + (t0 + t) * p.in_stride + r));
    th[i] = z;
  }
  __syncthreads();
  const bool on = c < p.d;
  const int64_t ch = (int64_t)h * p.d + (on ? c : 0);
  float z[DL_PREP_TOK];
  const float w0 = on ? p.w0[ch] : 0.f;
#pragma unroll
  for (int t = 0; t < DL_PREP_TOK; ++t) z[t] = w0;
  if (on) {
    const T* w2 = static_cast<const T*>(p.w2) + ch * p.w2_stride;   // rank padded to 4, zeros
    for (int r = 0; r < rank_p; r += 4) {
      const float4 w = Elem<T>::load4(w2 + r);
#pragma unroll
      for (int t = 0; t < DL_PREP_TOK; ++t) {
        const float4 x = *reinterpret_cast<const float4*>(th + t * rank_p + r);
        z[t] = fmaf(w.x, x.x, fmaf(w.y, x.y, fmaf(w.z, x.z, fmaf(w.w, x.w, z[t]))));
      }
    }
  }
  float kk[DL_PREP_TOK];
#pragma unroll
  for (int t = 0; t < DL_PREP_TOK; ++t) {
    kk[t] = on && t < nt
                ? Elem<T>::load(static_cast<const T*>(p.k) + (t0 + t) * p.in_stride + ch)
                : 0.f;
    const float s = warp_sum(kk[t] * kk[t]);
    if (lane == 0) ksq[warp * DL_PREP_TOK + t] = s;
  }
  __syncthreads();
  const float ab = on ? p.a_bias[ch] : 0.f;
#pragma unroll
  for (int t = 0; t < DL_PREP_TOK; ++t) {
    if (t >= nt) break;
    float s = 0.f;
    for (int i = 0; i < nwarps; ++i) s += ksq[i * DL_PREP_TOK + t];
    if (c < p.dp) {
      const int64_t row = (t0 + t) * p.in_stride + ch;
      float w = 0.f, u = 0.f, b = 0.f, r = 0.f, v = 0.f;
      if (on) {
        w = expf(-p.decay_scale * sigmoid_f32(z[t]));
        u = kk[t] * (1.0f / sqrtf(s + p.unit_eps));
        b = u * sigmoid_f32(Elem<T>::load(static_cast<const T*>(p.a) + row) + ab);
        r = Elem<T>::load(static_cast<const T*>(p.r) + row);
        v = Elem<T>::load(static_cast<const T*>(p.v) + row);
      }
      float* dst = p.packed + (((int64_t)h * p.rows + t0 + t) * DL_FIELDS) * p.dp + c;
      dst[0] = w;
      dst[p.dp] = u;
      dst[2 * p.dp] = b;
      dst[3 * p.dp] = kk[t];
      dst[4 * p.dp] = r;
      dst[5 * p.dp] = v;
    }
  }
}

struct DeltaScanParams {
  const float* packed;                 // [heads][rows][DL_FIELDS][dp]
  float* o;                            // [rows][heads * d]
  float* state;                        // [slots][heads][d][dp]
  const int32_t* cu; const int32_t* slots; const int64_t* positions;
  int64_t rows; int heads, d, dp, num_slots, num_portions;
  int tile;                            // tokens per stage
  int32_t* status;
};

// Packed pairs of fp32: one instruction, two IEEE multiply-adds.
__device__ __forceinline__ uint64_t dl_pack(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void dl_unpack(uint64_t v, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
}
__device__ __forceinline__ uint64_t dl_fma(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t dl_mul(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
// the 8 key channels of this thread: 4 * lane .. and 4 * (LANES + lane) ..
template <int LANES>
__device__ __forceinline__ void dl_load8(const float* row, int q, uint64_t (&x)[4]) {
  const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(row + q * 4);
  const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(row + (LANES + q) * 4);
  x[0] = a.x; x[1] = a.y; x[2] = b.x; x[3] = b.y;
}

// Thread = (column group, lane); NC columns per thread.  dp = 8 LANES.
template <int LANES, int NC>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_kernel(const DeltaScanParams p) {
  extern __shared__ __align__(128) uint8_t dl_smem[];
  constexpr int GROUPS = DL_THREADS / LANES;
  constexpr int COLS = GROUPS * NC;
  constexpr int DP = LANES * DL_CPL;
  constexpr int REC = DL_FIELDS * DP;         // floats per token
  const int stage_floats = p.tile * REC;
  float* stages = reinterpret_cast<float*>(dl_smem);
  float* outs = stages + DL_STAGES * stage_floats;                 // [2][tile][COLS]
  uint64_t* full = reinterpret_cast<uint64_t*>(outs + 2 * p.tile * COLS);
  __shared__ int failed;

  const int h = blockIdx.y, seq = blockIdx.z;
  const int col0 = blockIdx.x * COLS;
  const int q = threadIdx.x % LANES, grp = threadIdx.x / LANES;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < DL_STAGES; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
    failed = 0;
  }
  pdl_wait();
  const int64_t begin = p.cu[seq], end = p.cu[seq + 1];
  const int slot = begin < end ? p.slots[begin] : -1;
  const int64_t n = end - begin;
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
    return;
  }
  if (slot < 0 || n <= 0) return;
  __syncthreads();
  const int ntiles = (int)((n + p.tile - 1) / p.tile);
  const float* src = p.packed + ((int64_t)h * p.rows + begin) * REC;
  auto issue = [&](int tile_i) {
    const int s = tile_i % DL_STAGES;
    const int cnt = (int)min((int64_t)p.tile, n - (int64_t)tile_i * p.tile);
    const uint32_t bytes = (uint32_t)(cnt * REC * sizeof(float));
    mbar_arrive_expect_tx(&full[s], bytes);
    bulk_load(stages + s * stage_floats, src + (int64_t)tile_i * stage_floats, bytes, &full[s]);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < DL_STAGES - 1 && i < ntiles; ++i) issue(i);

  uint64_t s[NC][4];
  float* st[NC];
  bool col_on[NC];
  const bool fresh = p.positions[begin] == 0;
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    const int col = col0 + grp + j * GROUPS;
    col_on[j] = col < p.d;
    st[j] = p.state + (((int64_t)slot * p.heads + h) * p.d + (col_on[j] ? col : 0)) * DP;
#pragma unroll
    for (int i = 0; i < 4; ++i) s[j][i] = 0ull;
    if (col_on[j] && !fresh) dl_load8<LANES>(st[j], q, s[j]);
  }

  int ti = 0;
  for (; ti < ntiles; ++ti) {
    const int sg = ti % DL_STAGES;
    if (!mbar_wait(&full[sg], (uint32_t)(ti / DL_STAGES) & 1u, DL_WAIT_LIMIT)) {
      if (p.status) atomicOr(p.status, FK_DEV_WAIT_TIMEOUT);
      failed = 1;
    }
    const int cnt = (int)min((int64_t)p.tile, n - (int64_t)ti * p.tile);
    const float* rec = stages + sg * stage_floats;
    float* ot = outs + (ti & 1) * p.tile * COLS;
    for (int t = 0; t < cnt; ++t, rec += REC) {
      uint64_t w[4], u[4], b[4], k[4], r[4];
      dl_load8<LANES>(rec, q, w);
      dl_load8<LANES>(rec + DP, q, u);
      dl_load8<LANES>(rec + 2 * DP, q, b);
      dl_load8<LANES>(rec + 3 * DP, q, k);
      dl_load8<LANES>(rec + 4 * DP, q, r);
      float dot[NC], v[NC];
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        const int col = col0 + grp + j * GROUPS;
        v[j] = col < DP ? rec[5 * DP + col] : 0.f;
        const uint64_t d0 = dl_fma(u[1], s[j][1], dl_mul(u[0], s[j][0]));
        const uint64_t d1 = dl_fma(u[3], s[j][3], dl_mul(u[2], s[j][2]));
        float a0, a1, a2, a3;
        dl_unpack(d0, a0, a1);
        dl_unpack(d1, a2, a3);
        dot[j] = (a0 + a1) + (a2 + a3);
      }
      // the part of the update that does not wait for the reduction
      uint64_t nx[NC][4];
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        const uint64_t vv = dl_pack(v[j], v[j]);
#pragma unroll
        for (int i = 0; i < 4; ++i) nx[j][i] = dl_fma(k[i], vv, dl_mul(w[i], s[j][i]));
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1)
#pragma unroll
        for (int j = 0; j < NC; ++j) dot[j] += __shfl_xor_sync(0xffffffffu, dot[j], o);
      float out[NC];
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        const uint64_t nd = dl_pack(-dot[j], -dot[j]);
#pragma unroll
        for (int i = 0; i < 4; ++i) s[j][i] = dl_fma(b[i], nd, nx[j][i]);
        const uint64_t d0 = dl_fma(r[1], s[j][1], dl_mul(r[0], s[j][0]));
        const uint64_t d1 = dl_fma(r[3], s[j][3], dl_mul(r[2], s[j][2]));
        float a0, a1, a2, a3;
        dl_unpack(d0, a0, a1);
        dl_unpack(d1, a2, a3);
        out[j] = (a0 + a1) + (a2 + a3);
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1)
#pragma unroll
        for (int j = 0; j < NC; ++j) out[j] += __shfl_xor_sync(0xffffffffu, out[j], o);
      if (q == 0) {
#pragma unroll
        for (int j = 0; j < NC; ++j) ot[t * COLS + grp + j * GROUPS] = out[j];
      }
    }
    __syncthreads();   // stage sg is free, this tile's outputs are complete
    if (failed) break;
    if (threadIdx.x == 0 && ti + DL_STAGES - 1 < ntiles) issue(ti + DL_STAGES - 1);
    const int64_t row0 = begin + (int64_t)ti * p.tile;
    for (int i = threadIdx.x; i < cnt * COLS; i += DL_THREADS) {
      const int t = i / COLS, c = i - t * COLS;
      if (col0 + c < p.d)
        p.o[(row0 + t) * ((int64_t)p.heads * p.d) + (int64_t)h * p.d + col0 + c] = ot[i];
    }
  }
  if (failed) {
    // copies that were requested must land before the shared memory goes away
    for (int i = ti; i < ntiles && i < ti + DL_STAGES - 1; ++i)
      (void)mbar_wait(&full[i % DL_STAGES], (uint32_t)(i / DL_STAGES) & 1u, DL_WAIT_LIMIT);
    return;
  }
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    if (col_on[j]) {
      *reinterpret_cast<ulonglong2*>(st[j] + q * 4) = make_ulonglong2(s[j][0], s[j][1]);
      *reinterpret_cast<ulonglong2*>(st[j] + (LANES + q) * 4) = make_ulonglong2(s[j][2], s[j][3]);
    }
  }
}

struct DeltaOutParams {
  const float* o;                     // [rows][heads * d]
  const void* g; int64_t g_stride;    // gate projection
  const float* weight;                // [heads * d]
  void* out; int64_t out_stride;      // [rows, out_stride], tail beyond heads * d zeroed
  int64_t rows; int heads, d;
  float eps;
};

// One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) delta_output_kernel(const DeltaOutParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int64_t hd = (int64_t)p.heads * p.d;
  if (h > p.heads) return;
  for (int64_t t = blockIdx.y; t < p.rows; t += gridDim.y) {
    T* out = static_cast<T*>(p.out) + t * p.out_stride;
    if (h == p.heads) {
      for (int64_t c = hd + lane; c < p.out_stride; c += 32) Elem<T>::store(out + c, 0.f);
      continue;
    }
    const float* o = p.o + t * hd + (int64_t)h * p.d;
    const T* g = static_cast<const T*>(p.g) + t * p.g_stride + (int64_t)h * p.d;
    float x[DL_MAX_DIM / 32];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < DL_MAX_DIM / 32; ++i) {
      const int c = lane + i * 32;
      x[i] = c < p.d ? o[c] : 0.f;
      ss += x[i] * x[i];
    }
    ss = warp_sum(ss);
    const float rs = rsqrtf(ss / (float)p.d + p.eps);
#pragma unroll
    for (int i = 0; i < DL_MAX_DIM / 32; ++i) {
      const int c = lane + i * 32;
      if (c < p.d)
        Elem<T>::store(out + (int64_t)h * p.d + c,
                       x[i] * rs * p.weight[(int64_t)h * p.d + c] *
                           sigmoid_f32(Elem<T>::load(g + c)));
    }
  }
}

static int delta_lanes(int d) {
  return d <= 32 ? 4 : d <= 64 ? 8 : d <= 128 ? 16 : 32;
}

template <int LANES, int NC>
static int launch_scan(DeltaScanParams& p, cudaStream_t s) {
  constexpr int COLS = DL_THREADS / LANES * NC;
  constexpr int REC = DL_FIELDS * LANES * DL_CPL;
  // stage of at most 16 tokens and 24 KiB
  int tile = 16;
  while (tile > 4 && tile * REC * 4 > 24576) tile /= 2;
  p.tile = tile;
  const size_t smem = (size_t)DL_STAGES * tile * REC * 4 + 2ull * tile * COLS * 4 +
                      DL_STAGES * sizeof(uint64_t);
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, delta_scan_kernel<LANES, NC>, (int)smem));
  const dim3 grid((unsigned)((p.d + COLS - 1) / COLS), (unsigned)p.heads,
                  (unsigned)p.num_portions);
  FK_CUDA_OK(launch_kernel(delta_scan_kernel<LANES, NC>, grid, dim3(DL_THREADS), smem, s, p));
  count_launch();
  return FK_OK;
}
template <int LANES>
static int launch_scan_nc(DeltaScanParams& p, cudaStream_t s) {
  // two columns per thread keep the per-token chain short; with enough heads and
  // sequences to fill the SMs anyway, four halve the shared-memory reads
  const int64_t ctas2 = (int64_t)p.heads * p.num_portions *
                        ((p.d + DL_THREADS / LANES * 2 - 1) / (DL_THREADS / LANES * 2));
  if (ctas2 >= 4 * sm_count() && p.d > DL_THREADS / LANES * 2) return launch_scan<LANES, 4>(p, s);
  return launch_scan<LANES, 2>(p, s);
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_delta_padded_dim(int dim) {
  return dim <= 0 || dim > DL_MAX_DIM ? 0 : delta_lanes(dim) * DL_CPL;
}

int fk_delta_prepare(const void* r, const void* k, const void* v, const void* a, const void* y1,
                     int64_t in_stride, int is_f32, const void* w2, int64_t w2_stride,
                     const float* w0, const float* a_bias, float* packed, int64_t rows,
                     int heads, int dim, int rank, float decay_scale, float unit_eps,
                     fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && heads > 0 && dim > 0 && rank > 0, FK_ERR_INVALID_ARG,
             "fk_delta_prepare: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(r && k && v && a && y1 && w2 && w0 && a_bias && packed, FK_ERR_INVALID_ARG,
             "fk_delta_prepare: null pointer");
  FK_REQUIRE(dim <= DL_MAX_DIM && rank <= 512 && heads <= 65535, FK_ERR_UNSUPPORTED,
             "fk_delta_prepare: head size %d or rank %d too large", dim, rank);
  FK_REQUIRE(w2_stride % 4 == 0 && w2_stride >= rank && aligned16(w2) && aligned16(packed),
             FK_ERR_ALIGNMENT, "fk_delta_prepare: w2 rows must be padded to 4 elements");
  DeltaPrepParams p{};
  p.r = r; p.k = k; p.v = v; p.a = a; p.y1 = y1; p.in_stride = in_stride;
  p.w2 = w2; p.w2_stride = w2_stride; p.w0 = w0; p.a_bias = a_bias; p.packed = packed;
  p.rows = rows; p.heads = heads; p.d = dim; p.dp = fk_delta_padded_dim(dim); p.rank = rank;
  p.decay_scale = decay_scale; p.unit_eps = unit_eps;
  const int threads = p.dp;
  const size_t smem = (size_t)DL_PREP_TOK * ((rank + 3) / 4 * 4) * 4 +
                      (size_t)(threads / 32) * DL_PREP_TOK * 4;
  const dim3 grid((unsigned)((rows + DL_PREP_TOK - 1) / DL_PREP_TOK), (unsigned)heads);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32
                 ? launch_kernel(delta_prepare_kernel<float>, grid, dim3(threads), smem, s, p)
                 : launch_kernel(delta_prepare_kernel<uint16_t>, grid, dim3(threads), smem, s, p));
  count_launch();
  return FK_OK;
}

int fk_delta_scan(const float* packed, float* o, float* state, int num_slots,
                  const int32_t* cu_portions, int num_portions, const int32_t* slots,
                  const int64_t* positions, int64_t rows, int heads, int dim, int32_t* status,
                  fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && heads > 0 && dim > 0 && num_portions >= 0, FK_ERR_INVALID_ARG,
             "fk_delta_scan: bad sizes");
  if (rows == 0 || num_portions == 0) return FK_OK;
  FK_REQUIRE(packed && o && state && cu_portions && slots && positions && num_slots > 0,
             FK_ERR_INVALID_ARG, "fk_delta_scan: null pointer");
  FK_REQUIRE(dim <= DL_MAX_DIM && heads <= 65535 && num_portions <= 65535, FK_ERR_UNSUPPORTED,
             "fk_delta_scan: head size %d or counts too large", dim);
  FK_REQUIRE(aligned16(packed) && aligned16(state), FK_ERR_ALIGNMENT,
             "fk_delta_scan: 16-byte alignment required");
  DeltaScanParams p{};
  p.packed = packed; p.o = o; p.state = state; p.cu = cu_portions; p.slots = slots;
  p.positions = positions; p.rows = rows; p.heads = heads; p.d = dim;
  p.dp = fk_delta_padded_dim(dim); p.num_slots = num_slots; p.num_portions = num_portions;
  p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  switch (delta_lanes(dim)) {
    case 4: return launch_scan_nc<4>(p, s);
    case 8: return launch_scan_nc<8>(p, s);
    case 16: return launch_scan_nc<16>(p, s);
    default: return launch_scan_nc<32>(p, s);
  }
}

int fk_delta_output(const float* o, const void* gate, int64_t gate_stride, const float* weight,
                    void* out, int64_t out_stride, int is_f32, int64_t rows, int heads, int dim,
                    float eps, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && heads > 0 && dim > 0, FK_ERR_INVALID_ARG,
             "fk_delta_output: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(o && gate && weight && out, FK_ERR_INVALID_ARG, "fk_delta_output: null pointer");
  FK_REQUIRE(dim <= DL_MAX_DIM, FK_ERR_UNSUPPORTED, "fk_delta_output: head size %d too large",
             dim);
  FK_REQUIRE(out_stride >= (int64_t)heads * dim && gate_stride >= (int64_t)heads * dim,
             FK_ERR_INVALID_ARG, "fk_delta_output: bad stride");
  DeltaOutParams p{};
  p.o = o; p.g = gate; p.g_stride = gate_stride; p.weight = weight; p.out = out;
  p.out_stride = out_stride; p.rows = rows; p.heads = heads; p.d = dim; p.eps = eps;
  const dim3 grid((unsigned)(heads / 8 + 1), (unsigned)(rows < 8192 ? rows : 8192));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32 ? launch_kernel(delta_output_kernel<float>, grid, dim3(256), 0, s, p)
                    : launch_kernel(delta_output_kernel<uint16_t>, grid, dim3(256), 0, s, p));
  count_launch();
  return FK_OK;
}

}  // extern "C"
