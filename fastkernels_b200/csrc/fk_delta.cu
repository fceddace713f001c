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
//   delta_scan_blocked_kernel / delta_scan_kernel
//                          the recurrence.  The columns of S (value channels) are
//                          independent, so a column lives in the registers of LANES
//                          threads (8 key channels each); a CTA owns some columns of
//                          one head of one sequence.  Portions stream their packed
//                          tokens through a ring of shared-memory stages (bulk copies)
//                          and go four tokens at a time; single tokens are bound by
//                          the state's bytes.  The state comes from and returns to HBM
//                          once per call.
//   delta_output_kernel    per-head RMS norm of o, weight, output gate.
//
// State layout [slot][head][value channel][key channel (padded)], so that the
// threads of a column read 16-byte pieces that are adjacent across lanes.
#include "fk_types.cuh"

#include <cmath>

namespace fk {

constexpr int DL_FIELDS = 6;      // w, u, a * u, k, r, v
constexpr int DL_CPL = 8;         // key channels per thread
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

// What follows the decay projection, for one (token, channel).
template <typename T>
__device__ __forceinline__ void dl_pack_channel(const DeltaPrepParams& p, int64_t row, float z,
                                                float k, float unit, float a_bias, bool on,
                                                float* dst) {
  float w = 0.f, u = 0.f, b = 0.f, r = 0.f, v = 0.f;
  if (on) {
    w = expf(-p.decay_scale * sigmoid_f32(z));
    u = k * unit;
    b = u * sigmoid_f32(Elem<T>::load(static_cast<const T*>(p.a) + row) + a_bias);
    r = Elem<T>::load(static_cast<const T*>(p.r) + row);
    v = Elem<T>::load(static_cast<const T*>(p.v) + row);
  }
  dst[0] = w;
  dst[p.dp] = u;
  dst[2 * p.dp] = b;
  dst[3 * p.dp] = k;
  dst[4 * p.dp] = r;
  dst[5 * p.dp] = v;
}

// bf16: CTA = 16 tokens x one head at a time.  The decay projection runs on the
// tensor cores without losing the fp32 operand: tanh(y1) is split into two bf16 parts
// (16 significant bits; w2 is bf16 to begin with) and both products accumulate in
// fp32.  Then thread = (token, channel).
constexpr int DL_MMA_THREADS = 128;
__global__ void __launch_bounds__(DL_MMA_THREADS) delta_prepare_mma_kernel(
    const DeltaPrepParams p, int rank_p, int heads_per_cta) {
  extern __shared__ __align__(16) uint8_t dl_mma_smem[];
  pdl_launch_dependents();
  pdl_wait();
  // rows of 16-bit elements padded by 8 so that fragment loads hit different banks
  const int ld = rank_p + 8;
  uint16_t* hi = reinterpret_cast<uint16_t*>(dl_mma_smem);       // [16][ld]
  uint16_t* lo = hi + 16 * ld;                                   // [16][ld]
  float* zs = reinterpret_cast<float*>(lo + 16 * ld);            // [16][dp + 4]
  float* unit = zs + 16 * (p.dp + 4);                            // [16]
  const int zld = p.dp + 4;
  const int64_t t0 = (int64_t)blockIdx.x * 16;
  const int nt = (int)min((int64_t)16, p.rows - t0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int NW = DL_MMA_THREADS / 32;
  for (int i = threadIdx.x; i < 16 * rank_p; i += DL_MMA_THREADS) {
    const int t = i / rank_p, r = i - t * rank_p;
    float z = 0.f;
    if (t < nt && r < p.rank)
      z = tanhf(bf16_bits_to_float(
          static_cast<const uint16_t*>(p.y1)[(t0 + t) * p.in_stride + r]));
    const float zh = round_bf16(z);
    hi[t * ld + r] = __bfloat16_as_ushort(__float2bfloat16_rn(zh));
    lo[t * ld + r] = __bfloat16_as_ushort(__float2bfloat16_rn(z - zh));
  }
  const int h1 = min((int)(blockIdx.y + 1) * heads_per_cta, p.heads);
  for (int h = blockIdx.y * heads_per_cta; h < h1; ++h) {
    __syncthreads();       // tanh tile written; zs and unit of the last head consumed
    const int64_t ch0 = (int64_t)h * p.d;
    // 8 channels per step and warp: A = 16 tokens x rank, B = w2 rows (k contiguous)
    for (int n0 = warp * 8; n0 < p.d; n0 += NW * 8) {
      float c[4] = {0.f, 0.f, 0.f, 0.f};
      const int ch = n0 + (lane >> 2);
      const uint16_t* w2 = static_cast<const uint16_t*>(p.w2) +
                           (ch0 + (ch < p.d ? ch : 0)) * p.w2_stride;
      const int kq = (lane & 3) * 2, r0 = lane >> 2;
      for (int k0 = 0; k0 < rank_p; k0 += 16) {
        uint32_t b0 = 0, b1 = 0;
        if (ch < p.d) {
          if (k0 + kq < p.w2_stride) b0 = *reinterpret_cast<const uint32_t*>(w2 + k0 + kq);
          if (k0 + kq + 8 < p.w2_stride)
            b1 = *reinterpret_cast<const uint32_t*>(w2 + k0 + kq + 8);
        }
        const uint16_t* ah = hi + r0 * ld + k0 + kq;
        const uint16_t* al = lo + r0 * ld + k0 + kq;
        const uint32_t fh[4] = {*reinterpret_cast<const uint32_t*>(ah),
                                *reinterpret_cast<const uint32_t*>(ah + 8 * ld),
                                *reinterpret_cast<const uint32_t*>(ah + 8),
                                *reinterpret_cast<const uint32_t*>(ah + 8 * ld + 8)};
        const uint32_t fl[4] = {*reinterpret_cast<const uint32_t*>(al),
                                *reinterpret_cast<const uint32_t*>(al + 8 * ld),
                                *reinterpret_cast<const uint32_t*>(al + 8),
                                *reinterpret_cast<const uint32_t*>(al + 8 * ld + 8)};
        mma_bf16_16816(c, fl, b0, b1);
        mma_bf16_16816(c, fh, b0, b1);
      }
      const int cc = n0 + kq;      // this lane's two channels
      zs[r0 * zld + cc] = c[0];
      zs[r0 * zld + cc + 1] = c[1];
      zs[(r0 + 8) * zld + cc] = c[2];
      zs[(r0 + 8) * zld + cc + 1] = c[3];
    }
    // 1 / |k| of every token: warp w takes tokens w, w + NW, ...
    for (int t = warp; t < nt; t += NW) {
      const uint16_t* k = static_cast<const uint16_t*>(p.k) + (t0 + t) * p.in_stride + ch0;
      float s = 0.f;
      for (int c = lane; c < p.d; c += 32) {
        const float x = bf16_bits_to_float(k[c]);
        s += x * x;
      }
      s = warp_sum(s);
      if (lane == 0) unit[t] = 1.0f / sqrtf(s + p.unit_eps);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * p.dp; i += DL_MMA_THREADS) {
      const int t = i / p.dp, c = i - t * p.dp;
      const bool on = c < p.d;
      const int64_t row = (t0 + t) * p.in_stride + ch0 + c;
      const float k = on ? bf16_bits_to_float(static_cast<const uint16_t*>(p.k)[row]) : 0.f;
      dl_pack_channel<uint16_t>(p, row, on ? zs[t * zld + c] + p.w0[ch0 + c] : 0.f, k, unit[t],
                                on ? p.a_bias[ch0 + c] : 0.f, on,
                                p.packed + (((int64_t)h * p.rows + t0 + t) * DL_FIELDS) * p.dp + c);
    }
  }
}

// fp32: CTA = 16 tokens of one head, thread = key channel.
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
    dl_pack_channel<T>(p, (t0 + t) * p.in_stride + ch, z[t], kk[t],
                       1.0f / sqrtf(s + p.unit_eps), ab, on,
                       p.packed + (((int64_t)h * p.rows + t0 + t) * DL_FIELDS) * p.dp + c);
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

// One token of the recurrence for this thread's NC columns: s <- S_t, out = this
// lane's share of o_t.
template <int LANES, int NC>
__device__ __forceinline__ void dl_token(const float* rec, int q, int col0, int col_step,
                                         uint64_t (&s)[NC][4], float (&out)[NC]) {
  constexpr int DP = LANES * DL_CPL;
  uint64_t w[4], u[4], b[4], k[4], r[4];
  dl_load8<LANES>(rec + DP, q, u);
  dl_load8<LANES>(rec, q, w);
  dl_load8<LANES>(rec + 3 * DP, q, k);
  dl_load8<LANES>(rec + 2 * DP, q, b);
  dl_load8<LANES>(rec + 4 * DP, q, r);
  float dot[NC], v[NC];
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    const int col = col0 + j * col_step;
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
}

// Single tokens, or a handful: one token after the other.  Thread = (column group,
// lane); NC columns per thread, dp = 8 LANES.
template <int LANES, int NC, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_scan_kernel(const DeltaScanParams p) {
  constexpr int GROUPS = THREADS / LANES;
  constexpr int COLS = GROUPS * NC;
  constexpr int DP = LANES * DL_CPL;
  constexpr int REC = DL_FIELDS * DP;         // floats per token
  const int h = blockIdx.y, seq = blockIdx.z;
  const int col0 = blockIdx.x * COLS;
  const int q = threadIdx.x % LANES, grp = threadIdx.x / LANES;
  pdl_launch_dependents();
  pdl_wait();
  const int64_t begin = p.cu[seq], end = p.cu[seq + 1];
  const int slot = begin < end ? p.slots[begin] : -1;
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
    return;
  }
  if (slot < 0) return;
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
  for (int64_t t = begin; t < end; ++t) {
    float out[NC];
    dl_token<LANES, NC>(p.packed + ((int64_t)h * p.rows + t) * REC, q, col0 + grp, GROUPS, s,
                        out);
#pragma unroll
    for (int w = LANES / 2; w > 0; w >>= 1)
#pragma unroll
      for (int j = 0; j < NC; ++j) out[j] += __shfl_xor_sync(0xffffffffu, out[j], w);
    if (q == 0) {
#pragma unroll
      for (int j = 0; j < NC; ++j)
        if (col_on[j])
          p.o[t * ((int64_t)p.heads * p.d) + (int64_t)h * p.d + col0 + grp + j * GROUPS] = out[j];
    }
  }
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    if (col_on[j]) {
      *reinterpret_cast<ulonglong2*>(st[j] + q * 4) = make_ulonglong2(s[j][0], s[j][1]);
      *reinterpret_cast<ulonglong2*>(st[j] + (LANES + q) * 4) = make_ulonglong2(s[j][2], s[j][3]);
    }
  }
}

// Portions: four tokens at a time.  With S the state ahead of a block, u, b = a u, k,
// r, v of its tokens 1..4 and w_{j..i} = w_j ... w_i (elementwise),
//
//   p_i = u_i^T S_{i-1} = (u_i w_{1..i-1})^T S + sum_{j<i} A_ij v_j - C_ij p_j
//   o_i = S_i^T r_i     = (r_i w_{1..i})^T S   + sum_{j<=i} E_ij v_j - F_ij p_j
//   S_4 = w_{1..4} S + sum_j (k_j w_{j+1..4}) v_j^T - (b_j w_{j+1..4}) p_j^T
//   A_ij = u_i . (k_j w_{j+1..i-1}),  C: b for k,   E_ij = r_i . (k_j w_{j+1..i}),  F: b for k
//
// so a block has ONE reduction over a column's lanes on its critical path instead of
// four, and nothing is divided by a decay.  The scaled vectors and the 32 scalars do
// not depend on the state: the CTA works them out per stage, in place, before the
// column threads walk its blocks.  Missing tokens of a last block are w = 1 and zeros.
constexpr int DL_BLK = 4;
constexpr int DL_TILE = 16;           // tokens per stage
constexpr int DL_SCAL = 48;           // A (6) C (6) pad (4) | E 4x4 | F 4x4
constexpr int DL_SCAN_THREADS = 128;

template <int LANES, int NC>
__global__ void __launch_bounds__(DL_SCAN_THREADS) delta_scan_blocked_kernel(
    const DeltaScanParams p) {
  extern __shared__ __align__(128) uint8_t dl_smem[];
  constexpr int GROUPS = DL_SCAN_THREADS / LANES;
  constexpr int COLS = GROUPS * NC;
  constexpr int DP = LANES * DL_CPL;
  constexpr int REC = DL_FIELDS * DP;         // floats per token
  const int tile = p.tile;                    // a multiple of 4
  const int stage_floats = tile * REC;
  float* stages = reinterpret_cast<float*>(dl_smem);
  float* outs = stages + DL_STAGES * stage_floats;                 // [2][tile][COLS]
  float* scal = outs + 2 * tile * COLS;                            // [tile / 4][DL_SCAL]
  uint64_t* full = reinterpret_cast<uint64_t*>(scal + tile / DL_BLK * DL_SCAL);
  __shared__ int failed;

  const int h = blockIdx.y, seq = blockIdx.z;
  const int col0 = blockIdx.x * COLS;
  const int q = threadIdx.x % LANES, grp = threadIdx.x / LANES;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < DL_STAGES; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
    failed = 0;
  }
  for (int i = threadIdx.x; i < tile / DL_BLK * DL_SCAL; i += DL_SCAN_THREADS) scal[i] = 0.f;
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
  const int ntiles = (int)((n + tile - 1) / tile);
  const float* src = p.packed + ((int64_t)h * p.rows + begin) * REC;
  auto issue = [&](int tile_i) {
    const int s = tile_i % DL_STAGES;
    const int cnt = (int)min((int64_t)tile, n - (int64_t)tile_i * tile);
    const uint32_t bytes = (uint32_t)(cnt * REC * sizeof(float));
    mbar_arrive_expect_tx(&full[s], bytes);
    bulk_load(stages + s * stage_floats, src + (int64_t)tile_i * stage_floats, bytes, &full[s]);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < DL_STAGES - 1 && i < ntiles; ++i) issue(i);

  // where the scalar that this lane ends up with goes
  int scal_off = lane;
  if (lane >= 12) {
    const int e = lane - 12, f = e >= 10 ? 1 : 0, t = e - f * 10;
    const int row = t < 1 ? 0 : t < 3 ? 1 : t < 6 ? 2 : 3;
    scal_off = 16 + f * 16 + row * 4 + (t - row * (row + 1) / 2);
  }

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
    const int cnt = (int)min((int64_t)tile, n - (int64_t)ti * tile);
    const int blocks = (cnt + DL_BLK - 1) / DL_BLK;
    float* stage = stages + sg * stage_floats;
    // ---- state-free part: one warp per block, lane = channel
    for (int b = warp; b < blocks; b += DL_SCAN_THREADS / 32) {
      float acc[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) acc[i] = 0.f;
      for (int c = lane; c < DP; c += 32) {
        float* rec = stage + b * DL_BLK * REC + c;
        float kk[DL_BLK], bb[DL_BLK], gam = 1.f;
        int ia = 0, ie = 12;
#pragma unroll
        for (int i = 0; i < DL_BLK; ++i) {
          float* t = rec + i * REC;
          const bool on = b * DL_BLK + i < cnt;
          const float w = on ? t[0] : 1.f, u = on ? t[DP] : 0.f, r = on ? t[4 * DP] : 0.f;
#pragma unroll
          for (int j = 0; j < i; ++j) {
            acc[ia + j] = fmaf(u, kk[j], acc[ia + j]);
            acc[6 + ia + j] = fmaf(u, bb[j], acc[6 + ia + j]);
            kk[j] *= w;
            bb[j] *= w;
          }
          kk[i] = on ? t[3 * DP] : 0.f;
          bb[i] = on ? t[2 * DP] : 0.f;
#pragma unroll
          for (int j = 0; j <= i; ++j) {
            acc[ie + j] = fmaf(r, kk[j], acc[ie + j]);
            acc[10 + ie + j] = fmaf(r, bb[j], acc[10 + ie + j]);
          }
          ia += i;
          ie += i + 1;
          t[DP] = u * gam;
          gam *= w;
          t[4 * DP] = r * gam;
          if (!on) t[5 * DP] = 0.f;
        }
        rec[0] = gam;
#pragma unroll
        for (int j = 0; j < DL_BLK; ++j) {
          rec[j * REC + 3 * DP] = kk[j];
          rec[j * REC + 2 * DP] = bb[j];
        }
      }
      // 32 sums over the warp in 31 exchanges: lane l ends with sum number l
#pragma unroll
      for (int w = 16; w > 0; w >>= 1) {
        const bool up = (lane & w) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) {
          const float keep = up ? acc[i + w] : acc[i];
          const float give = up ? acc[i] : acc[i + w];
          acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
        }
      }
      scal[b * DL_SCAL + scal_off] = acc[0];
    }
    __syncthreads();
    // ---- the recurrence
    float* ot = outs + (ti & 1) * tile * COLS;
    for (int b = 0; b < blocks; ++b) {
      const float* rec = stage + b * DL_BLK * REC;
      const float* sc = scal + b * DL_SCAL;
      float v[DL_BLK][NC], d[DL_BLK][NC], o[DL_BLK][NC];
#pragma unroll
      for (int i = 0; i < DL_BLK; ++i) {
        uint64_t u[4];
        dl_load8<LANES>(rec + i * REC + DP, q, u);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const uint64_t x0 = dl_fma(u[1], s[j][1], dl_mul(u[0], s[j][0]));
          const uint64_t x1 = dl_fma(u[3], s[j][3], dl_mul(u[2], s[j][2]));
          float a0, a1, a2, a3;
          dl_unpack(x0, a0, a1);
          dl_unpack(x1, a2, a3);
          d[i][j] = (a0 + a1) + (a2 + a3);
        }
      }
#pragma unroll
      for (int w = LANES / 2; w > 0; w >>= 1)
#pragma unroll
        for (int i = 0; i < DL_BLK; ++i)
#pragma unroll
          for (int j = 0; j < NC; ++j) d[i][j] += __shfl_xor_sync(0xffffffffu, d[i][j], w);
      // off the critical path: output shares of the old state, decayed state, keys
#pragma unroll
      for (int i = 0; i < DL_BLK; ++i) {
        uint64_t r[4];
        dl_load8<LANES>(rec + i * REC + 4 * DP, q, r);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const uint64_t x0 = dl_fma(r[1], s[j][1], dl_mul(r[0], s[j][0]));
          const uint64_t x1 = dl_fma(r[3], s[j][3], dl_mul(r[2], s[j][2]));
          float a0, a1, a2, a3;
          dl_unpack(x0, a0, a1);
          dl_unpack(x1, a2, a3);
          o[i][j] = (a0 + a1) + (a2 + a3);
          const int col = col0 + grp + j * GROUPS;
          v[i][j] = col < DP ? rec[i * REC + 5 * DP + col] : 0.f;
        }
      }
      {
        uint64_t g[4];
        dl_load8<LANES>(rec, q, g);
#pragma unroll
        for (int j = 0; j < NC; ++j)
#pragma unroll
          for (int x = 0; x < 4; ++x) s[j][x] = dl_mul(g[x], s[j][x]);
      }
#pragma unroll
      for (int i = 0; i < DL_BLK; ++i) {
        uint64_t k[4];
        dl_load8<LANES>(rec + i * REC + 3 * DP, q, k);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const uint64_t vv = dl_pack(v[i][j], v[i][j]);
#pragma unroll
          for (int x = 0; x < 4; ++x) s[j][x] = dl_fma(k[x], vv, s[j][x]);
        }
      }
      // p_1 .. p_4 (kept in d)
      const float4 sa = *reinterpret_cast<const float4*>(sc);
      const float4 sb = *reinterpret_cast<const float4*>(sc + 4);
      const float4 sd = *reinterpret_cast<const float4*>(sc + 8);
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        d[1][j] += sa.x * v[0][j];
        d[2][j] += sa.y * v[0][j] + sa.z * v[1][j];
        d[3][j] += sa.w * v[0][j] + sb.x * v[1][j] + sb.y * v[2][j];
        d[1][j] -= sb.z * d[0][j];
        d[2][j] -= sb.w * d[0][j] + sd.x * d[1][j];
        d[3][j] -= sd.y * d[0][j] + sd.z * d[1][j] + sd.w * d[2][j];
      }
#pragma unroll
      for (int i = 0; i < DL_BLK; ++i) {
        uint64_t bv[4];
        dl_load8<LANES>(rec + i * REC + 2 * DP, q, bv);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const uint64_t np = dl_pack(-d[i][j], -d[i][j]);
#pragma unroll
          for (int x = 0; x < 4; ++x) s[j][x] = dl_fma(bv[x], np, s[j][x]);
        }
      }
      // outputs: lane i < 4 adds what the block's own tokens bring to token i, then the
      // shares are summed so that a lane ends with one token (its low two bits)
      const int row = q & 3;
      const float4 er = *reinterpret_cast<const float4*>(sc + 16 + row * 4);
      const float4 fr = *reinterpret_cast<const float4*>(sc + 32 + row * 4);
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        float corr = er.x * v[0][j] + er.y * v[1][j] + er.z * v[2][j] + er.w * v[3][j];
        corr -= fr.x * d[0][j] + fr.y * d[1][j] + fr.z * d[2][j] + fr.w * d[3][j];
#pragma unroll
        for (int i = 0; i < DL_BLK; ++i) o[i][j] += q == i ? corr : 0.f;
      }
#pragma unroll
      for (int w = 2; w > 0; w >>= 1) {
        const bool up = (q & w) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i)
#pragma unroll
          for (int j = 0; j < NC; ++j) {
            const float keep = up ? o[i + w][j] : o[i][j];
            const float give = up ? o[i][j] : o[i + w][j];
            o[i][j] = keep + __shfl_xor_sync(0xffffffffu, give, w);
          }
      }
#pragma unroll
      for (int w = LANES / 2; w >= 4; w >>= 1)
#pragma unroll
        for (int j = 0; j < NC; ++j) o[0][j] += __shfl_xor_sync(0xffffffffu, o[0][j], w);
      if (q < DL_BLK) {
#pragma unroll
        for (int j = 0; j < NC; ++j)
          ot[(b * DL_BLK + q) * COLS + grp + j * GROUPS] = o[0][j];
      }
    }
    fence_proxy_async_smem();   // the stage was rewritten in place; a copy comes next
    __syncthreads();            // stage sg is free, this tile's outputs are complete
    if (failed) break;
    if (threadIdx.x == 0 && ti + DL_STAGES - 1 < ntiles) issue(ti + DL_STAGES - 1);
    const int64_t row0 = begin + (int64_t)ti * tile;
    for (int i = threadIdx.x; i < cnt * COLS; i += DL_SCAN_THREADS) {
      const int t2 = i / COLS, c = i - t2 * COLS;
      if (col0 + c < p.d)
        p.o[(row0 + t2) * ((int64_t)p.heads * p.d) + (int64_t)h * p.d + col0 + c] = ot[i];
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

// d a multiple of 4: LPH lanes per (token, head), four channels a lane.
template <typename T, int LPH>
__global__ void __launch_bounds__(256) delta_output_vec_kernel(const DeltaOutParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int PER = 256 / LPH;                 // (token, head) pairs per CTA and pass
  const int j = threadIdx.x % LPH;
  const int h = blockIdx.x * PER + threadIdx.x / LPH;
  const int64_t hd = (int64_t)p.heads * p.d;
  const bool on = h < p.heads && j * 4 < p.d;
  const int64_t c0 = (int64_t)h * p.d + j * 4;
  const float4 wt = on ? __ldg(reinterpret_cast<const float4*>(p.weight + c0))
                       : make_float4(0.f, 0.f, 0.f, 0.f);
  for (int64_t t = blockIdx.y; t < p.rows; t += gridDim.y) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f), g = x;
    if (on) {
      x = *reinterpret_cast<const float4*>(p.o + t * hd + c0);
      g = Elem<T>::load4(static_cast<const T*>(p.g) + t * p.g_stride + c0);
    }
    float ss = sumsq(x);
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rs = rsqrtf(ss / (float)p.d + p.eps);
    T* out = static_cast<T*>(p.out) + t * p.out_stride;
    if (on)
      Elem<T>::store4(out + c0, (x * rs) * wt * make_float4(sigmoid_f32(g.x), sigmoid_f32(g.y),
                                                            sigmoid_f32(g.z), sigmoid_f32(g.w)));
    if (blockIdx.x == 0 && hd + threadIdx.x < p.out_stride && threadIdx.x < 64)
      Elem<T>::store(out + hd + threadIdx.x, 0.f);
  }
}

// One warp per (token, head), any d.
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

template <typename T, int LPH>
static cudaError_t launch_output_vec(const DeltaOutParams& p, cudaStream_t s) {
  constexpr int PER = 256 / LPH;
  const int gx = (p.heads + PER - 1) / PER;
  int64_t gy = (int64_t)sm_count() * 8 / gx;       // CTAs resident at once, tokens strided
  gy = gy < 1 ? 1 : gy < p.rows ? gy : p.rows;
  return launch_kernel(delta_output_vec_kernel<T, LPH>, dim3((unsigned)gx, (unsigned)gy),
                       dim3(256), 0, s, p);
}
template <typename T>
static cudaError_t launch_output(const DeltaOutParams& p, bool vec, cudaStream_t s) {
  if (vec && p.d <= 32) return launch_output_vec<T, 8>(p, s);
  if (vec && p.d <= 64) return launch_output_vec<T, 16>(p, s);
  if (vec) return launch_output_vec<T, 32>(p, s);
  const dim3 grid((unsigned)(p.heads / 8 + 1), (unsigned)(p.rows < 8192 ? p.rows : 8192));
  return launch_kernel(delta_output_kernel<T>, grid, dim3(256), 0, s, p);
}

static int delta_lanes(int d) {
  return d <= 32 ? 4 : d <= 64 ? 8 : d <= 128 ? 16 : 32;
}

template <int LANES, int NC>
static int launch_scan_blocked(DeltaScanParams& p, cudaStream_t s) {
  constexpr int COLS = DL_SCAN_THREADS / LANES * NC;
  constexpr int REC = DL_FIELDS * LANES * DL_CPL;
  int tile = DL_TILE;
  while (tile > DL_BLK && tile * REC * 4 > 24576) tile /= 2;
  p.tile = tile;
  const size_t smem = ((size_t)DL_STAGES * tile * REC + 2 * tile * COLS +
                       tile / DL_BLK * DL_SCAL) * 4 + DL_STAGES * sizeof(uint64_t);
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, delta_scan_blocked_kernel<LANES, NC>, (int)smem));
  const dim3 grid((unsigned)((p.d + COLS - 1) / COLS), (unsigned)p.heads,
                  (unsigned)p.num_portions);
  FK_CUDA_OK(launch_kernel(delta_scan_blocked_kernel<LANES, NC>, grid, dim3(DL_SCAN_THREADS), smem,
                           s, p));
  count_launch();
  return FK_OK;
}
template <int LANES>
static int launch_scan(DeltaScanParams& p, cudaStream_t s) {
  if (p.rows < 2 * (int64_t)p.num_portions) {    // (almost) all single tokens
    constexpr int COLS = 128 / LANES * 2;
    const dim3 grid((unsigned)((p.d + COLS - 1) / COLS), (unsigned)p.heads,
                    (unsigned)p.num_portions);
    FK_CUDA_OK(launch_kernel(delta_scan_kernel<LANES, 2, 128>, grid, dim3(128), 0, s, p));
    count_launch();
    return FK_OK;
  }
  // four columns per thread read the stage's vectors half as often as two, where
  // heads and sequences alone fill the SMs
  constexpr int COLS4 = DL_SCAN_THREADS / LANES * 4;
  if ((int64_t)p.heads * p.num_portions * ((p.d + COLS4 - 1) / COLS4) >= 2 * sm_count() &&
      p.d > COLS4 / 2)
    return launch_scan_blocked<LANES, 4>(p, s);
  return launch_scan_blocked<LANES, 2>(p, s);
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
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const unsigned tiles = (unsigned)((rows + DL_PREP_TOK - 1) / DL_PREP_TOK);
  if (is_f32) {
    const int threads = p.dp;
    const size_t smem = (size_t)DL_PREP_TOK * ((rank + 3) / 4 * 4) * 4 +
                        (size_t)(threads / 32) * DL_PREP_TOK * 4;
    FK_CUDA_OK(launch_kernel(delta_prepare_kernel<float>, dim3(tiles, (unsigned)heads),
                             dim3(threads), smem, s, p));
  } else {
    const int rank_p = (rank + 15) / 16 * 16;
    const size_t smem = 2ull * 16 * (rank_p + 8) * 2 + 16ull * (p.dp + 4) * 4 + 16 * 4;
    // heads per CTA: the tanh tile is shared by them, as long as the SMs stay busy
    int hpc = 1;
    while (hpc < 8 && (int64_t)tiles * heads / (hpc * 2) >= 16 * sm_count()) hpc *= 2;
    static PerDeviceOnce once;
    FK_CUDA_OK(set_max_dynamic_smem(once, delta_prepare_mma_kernel, 64 * 1024));
    FK_CUDA_OK(launch_kernel(delta_prepare_mma_kernel,
                             dim3(tiles, (unsigned)((heads + hpc - 1) / hpc)),
                             dim3(DL_MMA_THREADS), smem, s, p, rank_p, hpc));
  }
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
    case 4: return launch_scan<4>(p, s);
    case 8: return launch_scan<8>(p, s);
    case 16: return launch_scan<16>(p, s);
    default: return launch_scan<32>(p, s);
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
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = dim % 4 == 0 && dim <= 128 && gate_stride % 4 == 0 && out_stride % 4 == 0 &&
                   out_stride - (int64_t)heads * dim <= 64 && aligned16(o) && aligned16(gate) &&
                   aligned16(weight) && aligned16(out);
  FK_CUDA_OK(is_f32 ? launch_output<float>(p, vec, s) : launch_output<uint16_t>(p, vec, s));
  count_launch();
  return FK_OK;
}

}  // extern "C"
