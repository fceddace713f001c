// Generalized delta rule with a decay per key channel (linear attention with a
// matrix state per head), fp32 throughout:
//
//   S_t = diag(w_t) S_{t-1} - (a_t * u_t) (u_t^T S_{t-1}) + k_t v_t^T,   o_t = S_t^T r_t
//
//   w_t = exp(-c sigmoid(W2 tanh(y1) + w0)),  a_t = sigmoid(y_a + b_a),
//   u_t = k_t / sqrt(sum k_t^2 + eps_u)       (per head)
//
// Kernels:
//   delta_prepare_kernel        everything of a token that does not depend on the state:
//                               w, u, b = a * u, k, r, v as fp32, packed per (head, token);
//                               for portions in blocks of 4 tokens, with what the tokens
//                               of a block do to one another worked out (below)
//   delta_scan_kernel           the recurrence, token by token: single tokens, bound by
//                               the state's bytes
//   delta_scan_blocked_kernel   the recurrence over blocks, for portions
//
// The columns of S (value channels) are independent, so a column lives in the registers
// of LANES threads; a CTA owns some columns of one head of one sequence.  The state comes
// from and returns to HBM once per call, as [slot][head][value channel][key channel
// (padded)], so that the threads of a column read 16-byte pieces adjacent across lanes.
//
// Blocks.  With S the state ahead of a block, its tokens 1..4 and w_{j..i} = w_j ... w_i
// (elementwise):
//
//   p_i = u_i^T S_{i-1} = (u_i w_{1..i-1})^T S + sum_{j<i} A_ij v_j - C_ij p_j
//   o_i = S_i^T r_i     = (r_i w_{1..i})^T S   + sum_{j<=i} E_ij v_j - F_ij p_j
//   S_4 = w_{1..4} S + sum_j (k_j w_{j+1..4}) v_j^T - (b_j w_{j+1..4}) p_j^T
//   A_ij = u_i . (k_j w_{j+1..i-1}),  C: b for k,   E_ij = r_i . (k_j w_{j+1..i}),  F: b for k
//
// so a block has ONE reduction over a column's lanes on its critical path instead of
// four, and nothing is divided by a decay.  Missing tokens of a portion's last block are
// w = 1 and zeros.  A block is 21 dp + 48 floats:
//   u_i w_{1..i-1} [4][dp] | k_j w_{j+1..4} | -b_j w_{j+1..4} | r_i w_{1..i} | v_i |
//   w_{1..4} [dp] | A (6) C (6) pad (4) | E [4][4] | F [4][4]
// Blocks come in units of 16 tokens; portion i owns the units from cu[i] / 16 + i on.
#include "fk_types.cuh"

#include <cmath>

namespace fk {

constexpr int DL_FIELDS = 6;      // w, u, a * u, k, r, v
constexpr int DL_UNIT = 16;       // tokens per CTA of the prepare kernel
constexpr int DL_BLK = 4;         // tokens per block
constexpr int DL_STAGES = 3;
constexpr int DL_STAGE_BLOCKS = 2;
constexpr int DL_MAX_DIM = 256;
constexpr int DL_THREADS = 128;
constexpr uint32_t DL_WAIT_LIMIT = 1u << 20;
__host__ __device__ constexpr int dl_block_floats(int dp) { return 21 * dp + 48; }

struct DeltaPrepParams {
  const void* r; const void* k; const void* v; const void* a; const void* y1;
  int64_t in_stride;                    // packed projection rows
  const void* w2; int64_t w2_stride;    // [heads * d, rank]
  const float* w0; const float* a_bias; // [heads * d]
  float* packed;
  const int32_t* cu; int num_portions;  // blocks only
  int64_t rows, units; int heads, d, rank, rank_p, heads_per_cta;
  float decay_scale, unit_eps;
};

// fp32 exponential and sigmoid: the hardware approximations (relative error around
// 1e-6) beside bf16 operands, the accurate functions beside fp32 ones.
template <typename T>
struct Gate {
  static __device__ __forceinline__ float exp(float x) { return sizeof(T) == 2 ? __expf(x) : expf(x); }
  static __device__ __forceinline__ float sigmoid(float z) {
    return sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(-z)) : sigmoid_f32(z);
  }
};

// CTA = 16 tokens, some heads in turn.
template <typename T, int DP, bool BLOCKED>
__global__ void __launch_bounds__(DL_THREADS) delta_prepare_kernel(const DeltaPrepParams p) {
  extern __shared__ __align__(16) uint8_t dl_prep_smem[];
  pdl_launch_dependents();
  pdl_wait();
  constexpr bool MMA = sizeof(T) == 2;
  constexpr int NW = DL_THREADS / 32;
  int64_t t0 = (int64_t)blockIdx.x * DL_UNIT;
  int nt = (int)min((int64_t)DL_UNIT, p.rows - t0);
  if (BLOCKED) {
    int lo_i = 0, hi_i = p.num_portions;
    while (hi_i - lo_i > 1) {
      const int mid = (lo_i + hi_i) >> 1;
      if (p.cu[mid] / DL_UNIT + mid <= (int)blockIdx.x) lo_i = mid; else hi_i = mid;
    }
    t0 = p.cu[lo_i] + (int64_t)((int)blockIdx.x - (p.cu[lo_i] / DL_UNIT + lo_i)) * DL_UNIT;
    nt = (int)min((int64_t)DL_UNIT, (int64_t)p.cu[lo_i + 1] - t0);
  }
  if (nt <= 0) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  // tanh(y1): bf16 in two parts (w2 is bf16 to begin with, so the tensor cores keep 16
  // bits of the fp32 value and accumulate in fp32), fp32 as it is.  Rows of 16-bit
  // elements are padded by 8 so that fragment loads hit different banks.
  const int rank_p = p.rank_p, ld = rank_p + 8;
  uint16_t* hi = reinterpret_cast<uint16_t*>(dl_prep_smem);      // [16][ld] each
  uint16_t* lo = hi + DL_UNIT * ld;
  float* th = reinterpret_cast<float*>(dl_prep_smem);            // fp32: [16][rank_p]
  float* vec = reinterpret_cast<float*>(dl_prep_smem) + DL_UNIT * ld;   // [6][16][DP]
  float* part = vec + DL_FIELDS * DL_UNIT * DP;                  // [16][DP / 32]
  float* unit = part + DL_UNIT * (DP / 32);                      // [16]
  for (int i = threadIdx.x; i < DL_UNIT * rank_p; i += DL_THREADS) {
    const int t = i / rank_p, r = i - t * rank_p;
    float z = 0.f;
    if (t < nt && r < p.rank)
      z = tanhf(Elem<T>::load(static_cast<const T*>(p.y1) + (t0 + t) * p.in_stride + r));
    if (MMA) {
      const float zh = round_bf16(z);
      hi[t * ld + r] = __bfloat16_as_ushort(__float2bfloat16_rn(zh));
      lo[t * ld + r] = __bfloat16_as_ushort(__float2bfloat16_rn(z - zh));
    } else {
      th[i] = z;
    }
  }
  // where the sum that this lane ends up with goes inside a block's scalars
  int scal_off = lane;
  if (lane >= 12) {
    const int e = lane - 12, f = e >= 10 ? 1 : 0, t = e - f * 10;
    const int row = t < 1 ? 0 : t < 3 ? 1 : t < 6 ? 2 : 3;
    scal_off = 16 + f * 16 + row * 4 + (t - row * (row + 1) / 2);
  }
  const int h1 = min((int)(blockIdx.y + 1) * p.heads_per_cta, p.heads);
  for (int h = blockIdx.y * p.heads_per_cta; h < h1; ++h) {
    __syncthreads();       // tanh written; vec and unit of the last head consumed
    const int64_t ch0 = (int64_t)h * p.d;
    // this thread's elements of the head's [16][DP] tile.  Single tokens: requested before
    // the decay projection so that their latency passes behind it; blocks: as they are
    // needed, many CTAs share an SM
    constexpr int F = DL_UNIT * DP;                      // floats of one field
    constexpr int NIT = F / DL_THREADS;
    constexpr int PASS = BLOCKED ? 4 : NIT < 16 ? NIT : 16;
    constexpr int SL = DP / 32;                          // warps that hold one token
    // element x: token tok(x), channel chan(x); one channel per thread up to DP = 128
    constexpr int TSTEP = DP <= DL_THREADS ? DL_THREADS / DP : 1;
    constexpr int CPT = DP <= DL_THREADS ? 1 : DP / DL_THREADS;
    const int c_first = DP <= DL_THREADS ? (int)(threadIdx.x % DP) : (int)threadIdx.x;
    const int t_first = DP <= DL_THREADS ? (int)(threadIdx.x / DP) : 0;
    auto tok = [&](int x) { return t_first + x / CPT * TSTEP; };
    auto chan = [&](int x) { return c_first + x % CPT * DL_THREADS; };
    const int64_t base = (t0 + t_first) * p.in_stride + ch0 + c_first;
    const T* pk = static_cast<const T*>(p.k) + base;
    const T* pa = static_cast<const T*>(p.a) + base;
    const T* pr = static_cast<const T*>(p.r) + base;
    const T* pv = static_cast<const T*>(p.v) + base;
    auto offset = [&](int x) {
      return (int64_t)(x / CPT * TSTEP) * p.in_stride + x % CPT * DL_THREADS;
    };
    float w0c[CPT], abc[CPT];
#pragma unroll
    for (int x = 0; x < CPT; ++x) {
      const bool on = chan(x) < p.d;
      w0c[x] = on ? __ldg(p.w0 + ch0 + chan(x)) : 0.f;
      abc[x] = on ? __ldg(p.a_bias + ch0 + chan(x)) : 0.f;
    }
    T kx[PASS], ax[PASS], rx[PASS], vx[PASS];
    auto fetch = [&](int x0) {
#pragma unroll
      for (int x = 0; x < PASS; ++x) {
        kx[x] = ax[x] = rx[x] = vx[x] = T(0);
        if (tok(x0 + x) < nt && chan(x0 + x) < p.d) {
          const int64_t o = offset(x0 + x);
          kx[x] = __ldg(pk + o);
          ax[x] = __ldg(pa + o);
          rx[x] = __ldg(pr + o);
          vx[x] = __ldg(pv + o);
        }
      }
    };
    if (!BLOCKED) fetch(0);
    // decay projection into field 0
    if (MMA) {
      const int kq = (lane & 3) * 2, r0 = lane >> 2;
      for (int n0 = warp * 8; n0 < p.d; n0 += NW * 8) {
        float c[4] = {0.f, 0.f, 0.f, 0.f};
        const int ch = n0 + r0;
        const bool on = ch < p.d;
        const uint16_t* w2 = static_cast<const uint16_t*>(p.w2) + (ch0 + (on ? ch : 0)) * p.w2_stride;
        for (int k1 = 0; k1 < rank_p; k1 += 128) {
          uint32_t b0[8], b1[8];
#pragma unroll
          for (int x = 0; x < 8; ++x) {
            const int k0 = k1 + x * 16 + kq;
            b0[x] = b1[x] = 0u;
            if (on && k0 < p.w2_stride) b0[x] = __ldg(reinterpret_cast<const uint32_t*>(w2 + k0));
            if (on && k0 + 8 < p.w2_stride)
              b1[x] = __ldg(reinterpret_cast<const uint32_t*>(w2 + k0 + 8));
          }
#pragma unroll
          for (int x = 0; x < 8; ++x) {
            const int k0 = k1 + x * 16;
            if (k0 >= rank_p) break;
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
            mma_bf16_16816(c, fl, b0[x], b1[x]);
            mma_bf16_16816(c, fh, b0[x], b1[x]);
          }
        }
        *reinterpret_cast<float2*>(vec + r0 * DP + n0 + kq) = make_float2(c[0], c[1]);
        *reinterpret_cast<float2*>(vec + (r0 + 8) * DP + n0 + kq) = make_float2(c[2], c[3]);
      }
    } else {
      for (int i = threadIdx.x; i < nt * DP; i += DL_THREADS) {
        const int t = i / DP, c = i % DP;
        float z = 0.f;
        if (c < p.d) {
          const float* w2 = reinterpret_cast<const float*>(p.w2) + (ch0 + c) * p.w2_stride;
          for (int r = 0; r < p.rank; ++r) z = fmaf(w2[r], th[t * rank_p + r], z);
        }
        vec[i] = z;
      }
    }
    // sums of k^2 per token: [16][SL] partial sums, one per warp that holds some of it
#pragma unroll(BLOCKED ? 4 : NIT)
    for (int x = 0; x < NIT; ++x) {
      float k = 0.f;
      if (!BLOCKED && NIT <= PASS)
        k = Elem<T>::load(&kx[x < PASS ? x : 0]);
      else if (tok(x) < nt && chan(x) < p.d)
        k = Elem<T>::load(pk + offset(x));
      const float ss = warp_sum(k * k);
      if (lane == 0) part[tok(x) * SL + chan(x) / 32] = ss;
    }
    __syncthreads();
    if (threadIdx.x < DL_UNIT) {
      float ss = 0.f;
#pragma unroll
      for (int y = 0; y < SL; ++y) ss += part[threadIdx.x * SL + y];
      unit[threadIdx.x] = 1.0f / sqrtf(ss + p.unit_eps);
    }
    __syncthreads();
#pragma unroll(BLOCKED ? 1 : NIT / PASS)
    for (int x0 = 0; x0 < NIT; x0 += PASS) {
      if (BLOCKED || x0 > 0) fetch(x0);
#pragma unroll
      for (int x = 0; x < PASS; ++x) {
        const int t = tok(x0 + x), c = chan(x0 + x), i = t * DP + c;
        const bool on = t < nt && c < p.d;
        float w = 1.f, u = 0.f, b = 0.f;
        const float k = Elem<T>::load(&kx[x]), r = Elem<T>::load(&rx[x]);
        const float v = Elem<T>::load(&vx[x]);
        if (on) {
          w = Gate<T>::exp(-p.decay_scale * Gate<T>::sigmoid(vec[i] + w0c[x % CPT]));
          u = k * unit[t];
          b = u * Gate<T>::sigmoid(Elem<T>::load(&ax[x]) + abc[x % CPT]);
        }
        if (BLOCKED) {
          vec[i] = w;
          vec[F + i] = u;
          vec[2 * F + i] = b;
          vec[3 * F + i] = k;
          vec[4 * F + i] = r;
          vec[5 * F + i] = v;
        } else if (t < nt) {
          float* dst = p.packed + (((int64_t)h * p.rows + t0 + t) * DL_FIELDS) * DP + c;
          dst[0] = w;
          dst[DP] = u;
          dst[2 * DP] = b;
          dst[3 * DP] = k;
          dst[4 * DP] = r;
          dst[5 * DP] = v;
        }
      }
    }
    if (!BLOCKED) continue;
    __syncthreads();
    // a warp per block, lane = channel
    for (int blk = warp; blk * DL_BLK < nt; blk += NW) {
      float* dst = p.packed + (((int64_t)h * p.units + blockIdx.x) * (DL_UNIT / DL_BLK) + blk) *
                                  dl_block_floats(DP);
      float acc[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) acc[i] = 0.f;
#pragma unroll
      for (int c0 = 0; c0 < DP; c0 += 32) {
        const int c = c0 + lane;
        const float* src = vec + blk * DL_BLK * DP + c;
        float kk[DL_BLK], bb[DL_BLK], gam = 1.f;
#pragma unroll
        for (int i = 0; i < DL_BLK; ++i) {
          const int ia = i * (i - 1) / 2, ie = 12 + i * (i + 1) / 2;
          const float* s = src + i * DP;
          const float w = s[0], u = s[F], r = s[4 * F];
#pragma unroll
          for (int j = 0; j < i; ++j) {
            acc[ia + j] = fmaf(u, kk[j], acc[ia + j]);
            acc[6 + ia + j] = fmaf(u, bb[j], acc[6 + ia + j]);
            kk[j] *= w;
            bb[j] *= w;
          }
          bb[i] = s[2 * F];
          kk[i] = s[3 * F];
#pragma unroll
          for (int j = 0; j <= i; ++j) {
            acc[ie + j] = fmaf(r, kk[j], acc[ie + j]);
            acc[10 + ie + j] = fmaf(r, bb[j], acc[10 + ie + j]);
          }
          dst[i * DP + c] = u * gam;
          gam *= w;
          dst[(12 + i) * DP + c] = r * gam;
          dst[(16 + i) * DP + c] = s[5 * F];
        }
        dst[20 * DP + c] = gam;
#pragma unroll
        for (int j = 0; j < DL_BLK; ++j) {
          dst[(4 + j) * DP + c] = kk[j];
          dst[(8 + j) * DP + c] = -bb[j];
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
      float* scal = dst + 21 * DP;
      scal[16 + lane] = 0.f;           // E and F above their diagonals
      __syncwarp();
      scal[scal_off] = acc[0];
    }
  }
}

struct DeltaScanParams {
  const float* packed;                 // per token or blocks (see above)
  float* o;                            // [rows][heads * d]
  float* state;                        // [slots][heads][d][dp]
  const int32_t* cu; const int32_t* slots; const int64_t* positions;
  int64_t rows, units; int heads, d, num_slots, num_portions;
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
// The CPL key channels of lane q: 4 q .., 4 (LANES + q) .., ...
template <int LANES, int CPL>
__device__ __forceinline__ void dl_load(const float* row, int q, uint64_t (&x)[CPL / 2]) {
#pragma unroll
  for (int g = 0; g < CPL / 4; ++g) {
    const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(row + (g * LANES + q) * 4);
    x[2 * g] = a.x;
    x[2 * g + 1] = a.y;
  }
}
template <int LANES, int CPL>
__device__ __forceinline__ void dl_store(float* row, int q, const uint64_t (&x)[CPL / 2]) {
#pragma unroll
  for (int g = 0; g < CPL / 4; ++g)
    *reinterpret_cast<ulonglong2*>(row + (g * LANES + q) * 4) =
        make_ulonglong2(x[2 * g], x[2 * g + 1]);
}
__device__ __forceinline__ uint64_t dl_add(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
template <int N>
__device__ __forceinline__ float dl_dot(const uint64_t (&a)[N], const uint64_t (&b)[N]) {
  uint64_t x = dl_mul(a[0], b[0]);
  if (N > 2) {
    uint64_t y = dl_mul(a[1], b[1]);
#pragma unroll
    for (int i = 2; i < N; i += 2) {
      x = dl_fma(a[i], b[i], x);
      y = dl_fma(a[i + 1], b[i + 1], y);
    }
    x = dl_add(x, y);
  } else {
    x = dl_fma(a[N - 1], b[N - 1], x);
  }
  float a0, a1;
  dl_unpack(x, a0, a1);
  return a0 + a1;
}

// Token by token.  Thread = (column group, lane); NC columns per thread.
template <int LANES, int CPL, int NC>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_kernel(const DeltaScanParams p) {
  constexpr int GROUPS = DL_THREADS / LANES;
  constexpr int COLS = GROUPS * NC;
  constexpr int DP = LANES * CPL, NP = CPL / 2;
  constexpr int REC = DL_FIELDS * DP;         // floats per token
  const int h = blockIdx.y, seq = blockIdx.z;
  const int q = threadIdx.x % LANES, col0 = blockIdx.x * COLS + threadIdx.x / LANES;
  pdl_launch_dependents();
  pdl_wait();
  const int64_t begin = p.cu[seq], end = p.cu[seq + 1];
  const int slot = begin < end ? p.slots[begin] : -1;
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
    return;
  }
  if (slot < 0) return;
  uint64_t s[NC][NP];
  float* st[NC];
  bool col_on[NC];
  const bool fresh = p.positions[begin] == 0;
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    const int col = col0 + j * GROUPS;
    col_on[j] = col < p.d;
    st[j] = p.state + (((int64_t)slot * p.heads + h) * p.d + (col_on[j] ? col : 0)) * DP;
#pragma unroll
    for (int i = 0; i < NP; ++i) s[j][i] = 0ull;
    if (col_on[j] && !fresh) dl_load<LANES, CPL>(st[j], q, s[j]);
  }
  for (int64_t t = begin; t < end; ++t) {
    const float* rec = p.packed + ((int64_t)h * p.rows + t) * REC;
    uint64_t w[NP], u[NP], b[NP], k[NP], r[NP];
    dl_load<LANES, CPL>(rec + DP, q, u);
    dl_load<LANES, CPL>(rec, q, w);
    dl_load<LANES, CPL>(rec + 3 * DP, q, k);
    dl_load<LANES, CPL>(rec + 2 * DP, q, b);
    dl_load<LANES, CPL>(rec + 4 * DP, q, r);
    float dot[NC], out[NC];
#pragma unroll
    for (int j = 0; j < NC; ++j) dot[j] = dl_dot<NP>(u, s[j]);
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1)
#pragma unroll
      for (int j = 0; j < NC; ++j) dot[j] += __shfl_xor_sync(0xffffffffu, dot[j], o);
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      const int col = col0 + j * GROUPS;
      const float v = col < DP ? rec[5 * DP + col] : 0.f;
      const uint64_t vv = dl_pack(v, v), nd = dl_pack(-dot[j], -dot[j]);
#pragma unroll
      for (int i = 0; i < NP; ++i)
        s[j][i] = dl_fma(b[i], nd, dl_fma(k[i], vv, dl_mul(w[i], s[j][i])));
      out[j] = dl_dot<NP>(r, s[j]);
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1)
#pragma unroll
      for (int j = 0; j < NC; ++j) out[j] += __shfl_xor_sync(0xffffffffu, out[j], o);
    if (q == 0) {
#pragma unroll
      for (int j = 0; j < NC; ++j)
        if (col_on[j])
          p.o[t * ((int64_t)p.heads * p.d) + (int64_t)h * p.d + col0 + j * GROUPS] = out[j];
    }
  }
#pragma unroll
  for (int j = 0; j < NC; ++j)
    if (col_on[j]) dl_store<LANES, CPL>(st[j], q, s[j]);
}

// Blocks of a portion.  They stream through a ring of shared-memory stages (bulk
// copies); what limits the kernel is reading the blocks' vectors out of shared memory,
// which NC columns per thread share.
template <int LANES, int CPL, int NC>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_blocked_kernel(const DeltaScanParams p) {
  extern __shared__ __align__(128) uint8_t dl_smem[];
  constexpr int GROUPS = DL_THREADS / LANES;
  constexpr int COLS = GROUPS * NC;
  constexpr int DP = LANES * CPL, NP = CPL / 2;
  constexpr int BLK = DL_BLK, SB = DL_STAGE_BLOCKS;
  constexpr int REC = dl_block_floats(DP);    // floats per block
  float* stages = reinterpret_cast<float*>(dl_smem);
  float* outs = stages + DL_STAGES * SB * REC;                     // [2][SB * 4][COLS]
  uint64_t* full = reinterpret_cast<uint64_t*>(outs + 2 * SB * BLK * COLS);
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
  const int nblk = (int)((n + BLK - 1) / BLK);
  const int nst = (nblk + SB - 1) / SB;
  const float* src = p.packed + ((int64_t)h * p.units + begin / DL_UNIT + seq) *
                                    ((DL_UNIT / BLK) * (int64_t)REC);
  auto issue = [&](int si) {
    const int s = si % DL_STAGES;
    const uint32_t bytes = (uint32_t)(min(SB, nblk - si * SB) * REC * sizeof(float));
    mbar_arrive_expect_tx(&full[s], bytes);
    bulk_load(stages + s * SB * REC, src + (int64_t)si * SB * REC, bytes, &full[s]);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < DL_STAGES - 1 && i < nst; ++i) issue(i);

  uint64_t s[NC][NP];
  float* st[NC];
  bool col_on[NC];
  const bool fresh = p.positions[begin] == 0;
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    const int col = col0 + grp + j * GROUPS;
    col_on[j] = col < p.d;
    st[j] = p.state + (((int64_t)slot * p.heads + h) * p.d + (col_on[j] ? col : 0)) * DP;
#pragma unroll
    for (int i = 0; i < NP; ++i) s[j][i] = 0ull;
    if (col_on[j] && !fresh) dl_load<LANES, CPL>(st[j], q, s[j]);
  }

  int si = 0;
  for (; si < nst; ++si) {
    const int sg = si % DL_STAGES;
    if (!mbar_wait(&full[sg], (uint32_t)(si / DL_STAGES) & 1u, DL_WAIT_LIMIT)) {
      if (p.status) atomicOr(p.status, FK_DEV_WAIT_TIMEOUT);
      failed = 1;
    }
    const int blocks = min(SB, nblk - si * SB);
    float* ot = outs + (si & 1) * SB * BLK * COLS;
    for (int b = 0; b < blocks; ++b) {
      const float* rec = stages + (sg * SB + b) * REC;
      const float* sc = rec + 21 * DP;
      float v[BLK][NC], d[BLK][NC], o[BLK][NC];
#pragma unroll
      for (int i = 0; i < BLK; ++i) {
        uint64_t u[NP];
        dl_load<LANES, CPL>(rec + i * DP, q, u);
#pragma unroll
        for (int j = 0; j < NC; ++j) d[i][j] = dl_dot<NP>(u, s[j]);
      }
#pragma unroll
      for (int w = LANES / 2; w > 0; w >>= 1)
#pragma unroll
        for (int i = 0; i < BLK; i += 2)
#pragma unroll
          for (int j = 0; j < NC; ++j) {
            const float x0 = __shfl_xor_sync(0xffffffffu, d[i][j], w);
            const float x1 = __shfl_xor_sync(0xffffffffu, d[i + 1][j], w);
            dl_unpack(dl_add(dl_pack(d[i][j], d[i + 1][j]), dl_pack(x0, x1)), d[i][j],
                      d[i + 1][j]);
          }
      // off the critical path: output shares of the old state, decayed state, keys
#pragma unroll
      for (int i = 0; i < BLK; ++i) {
        uint64_t r[NP];
        dl_load<LANES, CPL>(rec + (12 + i) * DP, q, r);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          o[i][j] = dl_dot<NP>(r, s[j]);
          const int col = col0 + grp + j * GROUPS;
          v[i][j] = col < DP ? rec[(16 + i) * DP + col] : 0.f;
        }
      }
      {
        uint64_t g[NP];
        dl_load<LANES, CPL>(rec + 20 * DP, q, g);
#pragma unroll
        for (int j = 0; j < NC; ++j)
#pragma unroll
          for (int x = 0; x < NP; ++x) s[j][x] = dl_mul(g[x], s[j][x]);
      }
#pragma unroll
      for (int i = 0; i < BLK; ++i) {
        uint64_t k[NP];
        dl_load<LANES, CPL>(rec + (4 + i) * DP, q, k);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const uint64_t vv = dl_pack(v[i][j], v[i][j]);
#pragma unroll
          for (int x = 0; x < NP; ++x) s[j][x] = dl_fma(k[x], vv, s[j][x]);
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
      for (int i = 0; i < BLK; ++i) {
        uint64_t bv[NP];
        dl_load<LANES, CPL>(rec + (8 + i) * DP, q, bv);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const uint64_t np = dl_pack(d[i][j], d[i][j]);
#pragma unroll
          for (int x = 0; x < NP; ++x) s[j][x] = dl_fma(bv[x], np, s[j][x]);
        }
      }
      // outputs: halving exchanges over the low two lane bits leave token q & 3 in o[0],
      // then the sum over the other lanes and what the block's own tokens add
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
      for (int w = LANES / 2; w >= BLK; w >>= 1)
#pragma unroll
        for (int j = 0; j < NC; ++j) o[0][j] += __shfl_xor_sync(0xffffffffu, o[0][j], w);
      if (q < BLK) {
        const float4 er = *reinterpret_cast<const float4*>(sc + 16 + q * 4);
        const float4 fr = *reinterpret_cast<const float4*>(sc + 32 + q * 4);
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          const float x0 = er.x * v[0][j] + er.y * v[1][j] + er.z * v[2][j] + er.w * v[3][j];
          const float x1 = fr.x * d[0][j] + fr.y * d[1][j] + fr.z * d[2][j] + fr.w * d[3][j];
          ot[(b * BLK + q) * COLS + grp + j * GROUPS] = o[0][j] + (x0 - x1);
        }
      }
    }
    __syncthreads();            // stage sg is free, its outputs are complete
    if (failed) break;
    if (threadIdx.x == 0 && si + DL_STAGES - 1 < nst) issue(si + DL_STAGES - 1);
    const int64_t row0 = begin + (int64_t)si * SB * BLK;
    const int cnt = (int)min((int64_t)SB * BLK, end - row0);
    for (int i = threadIdx.x; i < cnt * COLS; i += DL_THREADS) {
      const int t2 = i / COLS, c = i - t2 * COLS;
      if (col0 + c < p.d)
        p.o[(row0 + t2) * ((int64_t)p.heads * p.d) + (int64_t)h * p.d + col0 + c] = ot[i];
    }
  }
  if (failed) {
    // copies that were requested must land before the shared memory goes away
    for (int i = si; i < nst && i < si + DL_STAGES - 1; ++i)
      (void)mbar_wait(&full[i % DL_STAGES], (uint32_t)(i / DL_STAGES) & 1u, DL_WAIT_LIMIT);
    return;
  }
#pragma unroll
  for (int j = 0; j < NC; ++j)
    if (col_on[j]) dl_store<LANES, CPL>(st[j], q, s[j]);
}

static int delta_padded(int d) { return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256; }

template <typename T, int DP, bool BLOCKED>
static int launch_prepare_one(const DeltaPrepParams& p, unsigned gx, cudaStream_t s) {
  const size_t smem = (size_t)DL_UNIT * (p.rank_p + 8) * 4 +
                      (size_t)DL_FIELDS * DL_UNIT * DP * 4 + DL_UNIT * (DP / 32 + 1) * 4;
  static PerDeviceOnce once;
  constexpr int kMaxSmem = DL_UNIT * 520 * 4 + DL_FIELDS * DL_UNIT * DP * 4 +
                           DL_UNIT * (DP / 32 + 1) * 4;
  FK_CUDA_OK(set_max_dynamic_smem(once, delta_prepare_kernel<T, DP, BLOCKED>, kMaxSmem));
  const dim3 grid(gx, (unsigned)((p.heads + p.heads_per_cta - 1) / p.heads_per_cta));
  FK_CUDA_OK(launch_kernel(delta_prepare_kernel<T, DP, BLOCKED>, grid, dim3(DL_THREADS), smem, s,
                           p));
  count_launch();
  return FK_OK;
}
template <typename T, int DP>
static int launch_prepare_dp(const DeltaPrepParams& p, bool blocked, cudaStream_t s) {
  if (blocked) return launch_prepare_one<T, DP, true>(p, (unsigned)p.units, s);
  return launch_prepare_one<T, DP, false>(p, (unsigned)((p.rows + DL_UNIT - 1) / DL_UNIT), s);
}
template <typename T>
static int launch_prepare(const DeltaPrepParams& p, bool blocked, cudaStream_t s) {
  switch (delta_padded(p.d)) {
    case 32: return launch_prepare_dp<T, 32>(p, blocked, s);
    case 64: return launch_prepare_dp<T, 64>(p, blocked, s);
    case 128: return launch_prepare_dp<T, 128>(p, blocked, s);
    default: return launch_prepare_dp<T, 256>(p, blocked, s);
  }
}

template <int LANES, int CPL, int NC>
static int launch_scan_blocked(DeltaScanParams& p, cudaStream_t s) {
  constexpr int COLS = DL_THREADS / LANES * NC;
  constexpr size_t kSmem = ((size_t)DL_STAGES * DL_STAGE_BLOCKS * dl_block_floats(LANES * CPL) +
                            2 * DL_STAGE_BLOCKS * DL_BLK * COLS) * 4 +
                           DL_STAGES * sizeof(uint64_t);
  static PerDeviceOnce once;
  FK_CUDA_OK(set_max_dynamic_smem(once, delta_scan_blocked_kernel<LANES, CPL, NC>, (int)kSmem));
  const dim3 grid((unsigned)((p.d + COLS - 1) / COLS), (unsigned)p.heads,
                  (unsigned)p.num_portions);
  // not ahead of its predecessor's end: CTAs that squeeze in beside the last ones of it
  // pile up on a few SMs and stay there
  FK_CUDA_OK(launch_kernel_after(delta_scan_blocked_kernel<LANES, CPL, NC>, grid,
                                 dim3(DL_THREADS), kSmem, s, p));
  count_launch();
  return FK_OK;
}
// LANES x CPL for single tokens, BL x BC for blocks
template <int LANES, int CPL, int BL, int BC>
static int launch_scan(DeltaScanParams& p, bool blocked, cudaStream_t s) {
  if (!blocked) {
    constexpr int COLS = DL_THREADS / LANES * 2;
    const dim3 grid((unsigned)((p.d + COLS - 1) / COLS), (unsigned)p.heads,
                    (unsigned)p.num_portions);
    FK_CUDA_OK(launch_kernel(delta_scan_kernel<LANES, CPL, 2>, grid, dim3(DL_THREADS), 0, s, p));
    count_launch();
    return FK_OK;
  }
  // four columns per thread read a stage's vectors half as often as two; two make a
  // block's instructions fewer where small heads and few sequences do not fill the SMs
  constexpr int COLS4 = DL_THREADS / BL * 4;
  if (p.d > 64 || (p.d > COLS4 / 2 && (int64_t)p.heads * p.num_portions *
                                              ((p.d + COLS4 - 1) / COLS4) >= 2 * sm_count()))
    return launch_scan_blocked<BL, BC, 4>(p, s);
  return launch_scan_blocked<BL, BC, 2>(p, s);
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_delta_padded_dim(int dim) {
  return dim <= 0 || dim > DL_MAX_DIM ? 0 : delta_padded(dim);
}

int64_t fk_delta_packed_floats(int64_t rows, int num_portions, int heads, int dim, int blocked) {
  const int dp = fk_delta_padded_dim(dim);
  if (dp == 0 || rows < 0 || num_portions < 0 || heads <= 0) return 0;
  return blocked ? heads * (rows / DL_UNIT + num_portions) * (DL_UNIT / DL_BLK) *
                       (int64_t)dl_block_floats(dp)
                 : heads * rows * (int64_t)DL_FIELDS * dp;
}

int fk_delta_prepare(const void* r, const void* k, const void* v, const void* a, const void* y1,
                     int64_t in_stride, int is_f32, const void* w2, int64_t w2_stride,
                     const float* w0, const float* a_bias, float* packed, int blocked,
                     const int32_t* cu_portions, int num_portions, int64_t rows,
                     int heads, int dim, int rank, float decay_scale, float unit_eps,
                     fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && heads > 0 && dim > 0 && rank > 0, FK_ERR_INVALID_ARG,
             "fk_delta_prepare: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(r && k && v && a && y1 && w2 && w0 && a_bias && packed, FK_ERR_INVALID_ARG,
             "fk_delta_prepare: null pointer");
  FK_REQUIRE(!blocked || (cu_portions && num_portions > 0), FK_ERR_INVALID_ARG,
             "fk_delta_prepare: blocks need the portions");
  FK_REQUIRE(dim <= DL_MAX_DIM && rank <= 512 && heads <= 65535 && rows < (1ll << 31),
             FK_ERR_UNSUPPORTED, "fk_delta_prepare: head size %d or rank %d too large", dim, rank);
  FK_REQUIRE(w2_stride % 4 == 0 && w2_stride >= rank && aligned16(w2) && aligned16(packed),
             FK_ERR_ALIGNMENT, "fk_delta_prepare: w2 rows must be padded to 4 elements");
  DeltaPrepParams p{};
  p.r = r; p.k = k; p.v = v; p.a = a; p.y1 = y1; p.in_stride = in_stride;
  p.w2 = w2; p.w2_stride = w2_stride; p.w0 = w0; p.a_bias = a_bias; p.packed = packed;
  p.cu = cu_portions; p.num_portions = num_portions;
  p.rows = rows; p.units = rows / DL_UNIT + num_portions;
  p.heads = heads; p.d = dim; p.rank = rank; p.rank_p = (rank + 15) / 16 * 16;
  p.decay_scale = decay_scale; p.unit_eps = unit_eps;
  // heads per CTA: the tanh tile is shared by them, as long as the SMs stay busy
  int hpc = 1;
  while (hpc < 8 && (rows / DL_UNIT + 1) * heads / (hpc * 2) >= 16 * sm_count()) hpc *= 2;
  p.heads_per_cta = hpc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return is_f32 ? launch_prepare<float>(p, blocked != 0, s)
                : launch_prepare<uint16_t>(p, blocked != 0, s);
}

int fk_delta_scan(const float* packed, int blocked, float* o, float* state, int num_slots,
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
  p.positions = positions; p.rows = rows; p.units = rows / DL_UNIT + num_portions;
  p.heads = heads; p.d = dim; p.num_slots = num_slots; p.num_portions = num_portions;
  p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  switch (delta_padded(dim)) {
    case 32: return launch_scan<4, 8, 4, 8>(p, blocked != 0, s);
    case 64: return launch_scan<8, 8, 8, 8>(p, blocked != 0, s);
    case 128: return launch_scan<16, 8, 16, 8>(p, blocked != 0, s);
    default: return launch_scan<32, 8, 32, 8>(p, blocked != 0, s);
  }
}

}  // extern "C"
