// Matrix memory (mLSTM): per head a matrix S [dim, vdim], a vector n [dim] and a running
// maximum m, all fp32, with log gates i and f per token:
//
//   i = cap tanh(zi / cap), f = logsigmoid(cap tanh(zf / cap))
//   m' = max(f + m, i),  S' = e^{f + m - m'} S + e^{i - m'} k v^T,  n' alike with k
//   o = S'^T q / (max(|n' . q|, e^{-m'}) + 1e-6),   m = 0 at the start
//
//   mlstm_step_kernel     one token per sequence: state streamed once, head norm and
//                         output gate applied on the way out
//   mlstm_scan_kernel     portions, token by token, any size, bf16 or fp32
//   chunked form (bf16)   blocks ("units") of 128 tokens of a portion.  With g_t the sum of
//                         f inside the unit up to t and S, n, m the values ahead of it,
//     m_t   = max(g_t + m, max_{s <= t} g_t - g_s + i_s)
//     num_t = e^{g_t + m - m_t} S^T q_t + sum_{s <= t} e^{g_t - g_s + i_s - m_t} (q_t . k_s) v_s
//   mlstm_gates_kernel    gates, g, m of every token, decay of every unit
//   mlstm_unit_kernel     what a unit adds to S and n                     (tensor cores)
//   mlstm_carry_kernel    S and n ahead of every unit: a scan over units, per element
//   mlstm_output_kernel   num / denominator                               (tensor cores)
// Units are counted from the start of a portion, which changes results by rounding only.
// fp32 operands of the tensor products (decayed v, S, decayed scores) enter as two bf16
// parts, 16 significant bits; q, k, v are bf16 projections.
#include "fk_types.cuh"

#include <cmath>

namespace fk {

constexpr int ML_UNIT = 128;
constexpr float ML_EPS = 1e-6f;
constexpr float ML_NONE = -1e30f;     // log gate of a token that is not there

struct MlstmParams {
  const void* q; const void* k; const void* v; int64_t in_stride;   // packed projection rows
  const float* z; int64_t z_stride;            // [rows, 2 heads]: input, forget
  float* s_state; float* n_state;              // [slots, heads, dim, vp], [slots, heads, np]
  int num_slots;
  const int32_t* cu; int num_portions;
  const int32_t* slots; const int64_t* positions;
  int64_t rows, units; int most_units;
  int heads, dim, vdim, vp, np;                // n_state: n at 0 .. dim - 1, m at dim
  float cap, q_scale;
  // step only
  const void* gate; int64_t gate_stride; const float* weight; float eps;
  void* out; int64_t out_stride;
  // portions
  float* o;                                    // [rows, heads * vdim]
  float* gg; float* gi; float* gm;             // [heads][units * ML_UNIT]: g, i, m
  float* unit_m; float* unit_decay;            // [heads][units]
  float* inc;                                  // [units][heads][dim][vp]
  float* ninc;                                 // [units][heads][dim]
  int32_t* status;
};

__device__ __forceinline__ float ml_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_forget_gate(float z, float cap) {
  const float u = cap * tanhf(z / cap);
  return fminf(u, 0.f) - log1pf(expf(-fabsf(u)));
}
__device__ __forceinline__ bool ml_slot_ok(const MlstmParams& p, int slot) {
  if (slot >= p.num_slots && threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
  return slot >= 0 && slot < p.num_slots;
}

// ------------------------------------------------------------------ one token a sequence
constexpr int MS_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(MS_THREADS) mlstm_step_kernel(const MlstmParams p) {
  extern __shared__ float ms_smem[];           // q [dim] | k [dim] | partial o [groups][vp]
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[64];
  int flip = 0;
  const int h = blockIdx.x, tid = threadIdx.x;
  const int64_t t = blockIdx.y;
  T* out = static_cast<T*>(p.out) + t * p.out_stride;
  const int hv = p.heads * p.vdim;
  if (h == 0)
    for (int c = hv + tid; c < p.out_stride; c += MS_THREADS) Elem<T>::store(out + c, 0.f);
  const int slot = p.slots[t];
  if (!ml_slot_ok(p, slot)) {
    for (int c = tid; c < p.vdim; c += MS_THREADS) Elem<T>::store(out + h * p.vdim + c, 0.f);
    return;
  }
  float* qs = ms_smem;
  const int dim4 = (p.dim + 3) & ~3;
  float* ks = qs + dim4;
  float* part = ks + dim4;
  const T* q = static_cast<const T*>(p.q) + t * p.in_stride + h * p.dim;
  const T* k = static_cast<const T*>(p.k) + t * p.in_stride + h * p.dim;
  const T* v = static_cast<const T*>(p.v) + t * p.in_stride + h * p.vdim;
  float* S = p.s_state + ((int64_t)slot * p.heads + h) * p.dim * p.vp;
  float* N = p.n_state + ((int64_t)slot * p.heads + h) * p.np;
  const bool fresh = p.positions[t] == 0;
  const float m_old = fresh ? 0.f : N[p.dim];
  const float gi = ml_input_gate(p.z[t * p.z_stride + h], p.cap);
  const float gf = ml_forget_gate(p.z[t * p.z_stride + p.heads + h], p.cap);
  const float m = fmaxf(gf + m_old, gi);
  const float keep = fresh ? 0.f : expf(gf + m_old - m), add = expf(gi - m);
  float nq[1] = {0.f};
  for (int c = tid; c < p.dim; c += MS_THREADS) {
    const float kc = Elem<T>::load(k + c), qc = Elem<T>::load(q + c) * p.q_scale;
    ks[c] = kc * add;
    qs[c] = qc;
    const float n = (fresh ? 0.f : keep * N[c]) + add * kc;
    N[c] = n;
    nq[0] += n * qc;
  }
  block_sums<1>(nq, red, flip);                // also: ks, qs written; m_old read by all
  if (tid == 0) N[p.dim] = m;
  const int cgs = p.vp >> 2, groups = MS_THREADS / cgs;
  const int cg = tid % cgs, rg = tid / cgs;
  if (rg < groups) {
    const int c0 = cg * 4;
    const float4 vv = make_float4(c0 < p.vdim ? Elem<T>::load(v + c0) : 0.f,
                                  c0 + 1 < p.vdim ? Elem<T>::load(v + c0 + 1) : 0.f,
                                  c0 + 2 < p.vdim ? Elem<T>::load(v + c0 + 2) : 0.f,
                                  c0 + 3 < p.vdim ? Elem<T>::load(v + c0 + 3) : 0.f);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr int UN = 8;
    for (int r0 = rg; r0 < p.dim; r0 += groups * UN) {
      float4 s[UN];
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int r = r0 + u * groups;
        s[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < p.dim && !fresh)
          s[u] = *reinterpret_cast<const float4*>(S + (int64_t)r * p.vp + c0);
      }
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int r = r0 + u * groups;
        if (r < p.dim) {
          s[u] = s[u] * keep + vv * ks[r];
          *reinterpret_cast<float4*>(S + (int64_t)r * p.vp + c0) = s[u];
          acc = acc + s[u] * qs[r];
        }
      }
    }
    *reinterpret_cast<float4*>(part + rg * p.vp + c0) = acc;
  }
  __syncthreads();
  const float inv = 1.0f / (fmaxf(fabsf(nq[0]), expf(-m)) + ML_EPS);
  float ss[1] = {0.f};
  for (int c = tid; c < p.vdim; c += MS_THREADS) {
    float x = 0.f;
    for (int g = 0; g < groups; ++g) x += part[g * p.vp + c];
    x *= inv;
    part[c] = x;                               // own column of group 0: read above by this thread
    ss[0] += x * x;
  }
  block_sums<1>(ss, red, flip);
  const float rs = rsqrtf(ss[0] / (float)p.vdim + p.eps);
  const T* gt = static_cast<const T*>(p.gate) + t * p.gate_stride + h * p.vdim;
  for (int c = tid; c < p.vdim; c += MS_THREADS)
    Elem<T>::store(out + h * p.vdim + c, part[c] * rs * p.weight[h * p.vdim + c] *
                                             sigmoid_f32(Elem<T>::load(gt + c)));
}

// ----------------------------------------------------------------- portions, any size
constexpr int MC_COLS = 32, MC_GROUPS = 4;
template <typename T>
__global__ void __launch_bounds__(MC_COLS * MC_GROUPS) mlstm_scan_kernel(const MlstmParams p) {
  extern __shared__ float mc_smem[];    // S [dim][32] | n [dim] | q [2][dim] | k [2][dim]
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[64], part[2][MC_GROUPS][MC_COLS];
  int flip = 0;
  const int h = blockIdx.y, pi = blockIdx.z, tid = threadIdx.x;
  const int64_t t0 = p.cu[pi], t1 = min((int64_t)p.cu[pi + 1], p.rows);
  if (t0 < 0 || t0 >= t1) return;
  const int slot = p.slots[t0];
  const bool keep_state = ml_slot_ok(p, slot);
  const int col = tid % MC_COLS, rg = tid / MC_COLS;
  const int c = blockIdx.x * MC_COLS + col;
  const bool on = c < p.vdim;
  float* S = mc_smem;
  float* n = S + p.dim * MC_COLS;
  float* qs = n + p.dim;
  float* ks = qs + 2 * p.dim;
  const int64_t at = keep_state ? slot : 0;
  float* gS = p.s_state + (at * p.heads + h) * p.dim * p.vp;
  float* gN = p.n_state + (at * p.heads + h) * p.np;
  const bool load = keep_state && p.positions[t0] > 0;
  for (int r = rg; r < p.dim; r += MC_GROUPS)
    S[r * MC_COLS + col] = load && on ? gS[(int64_t)r * p.vp + c] : 0.f;
  for (int r = tid; r < p.dim; r += blockDim.x) n[r] = load ? gN[r] : 0.f;
  float m = load ? gN[p.dim] : 0.f;
  for (int64_t t = t0; t < t1; ++t) {
    const int b = (int)(t & 1);
    const float gi = ml_input_gate(p.z[t * p.z_stride + h], p.cap);
    const float gf = ml_forget_gate(p.z[t * p.z_stride + p.heads + h], p.cap);
    const float m2 = fmaxf(gf + m, gi);
    const float keep = expf(gf + m - m2), add = expf(gi - m2);
    m = m2;
    const T* q = static_cast<const T*>(p.q) + t * p.in_stride + h * p.dim;
    const T* k = static_cast<const T*>(p.k) + t * p.in_stride + h * p.dim;
    float nq[1] = {0.f};
    for (int r = tid; r < p.dim; r += blockDim.x) {
      const float kc = Elem<T>::load(k + r), qc = Elem<T>::load(q + r) * p.q_scale;
      qs[b * p.dim + r] = qc;
      ks[b * p.dim + r] = kc * add;
      n[r] = keep * n[r] + add * kc;
      nq[0] += n[r] * qc;
    }
    block_sums<1>(nq, red, flip);
    const float vv = on ? Elem<T>::load(static_cast<const T*>(p.v) + t * p.in_stride +
                                        h * p.vdim + c) : 0.f;
    float acc = 0.f;
    for (int r = rg; r < p.dim; r += MC_GROUPS) {
      const float s = keep * S[r * MC_COLS + col] + ks[b * p.dim + r] * vv;
      S[r * MC_COLS + col] = s;
      acc = fmaf(s, qs[b * p.dim + r], acc);
    }
    part[b][rg][col] = acc;
    __syncthreads();
    if (rg == 0 && on) {
      float o = 0.f;
#pragma unroll
      for (int g = 0; g < MC_GROUPS; ++g) o += part[b][g][col];
      p.o[t * ((int64_t)p.heads * p.vdim) + h * p.vdim + c] =
          o / (fmaxf(fabsf(nq[0]), expf(-m)) + ML_EPS);
    }
  }
  if (!keep_state) return;
  for (int r = rg; r < p.dim; r += MC_GROUPS)
    if (on) gS[(int64_t)r * p.vp + c] = S[r * MC_COLS + col];
}

// n and m after the portions, for the scan: several CTAs of a head read the old values, so
// they are written by a launch of their own.
template <typename T>
__global__ void __launch_bounds__(128) mlstm_scan_norm_kernel(const MlstmParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, pi = blockIdx.y;
  const int64_t t0 = p.cu[pi], t1 = min((int64_t)p.cu[pi + 1], p.rows);
  if (t0 < 0 || t0 >= t1) return;
  const int slot = p.slots[t0];
  if (!ml_slot_ok(p, slot)) return;
  float* gN = p.n_state + ((int64_t)slot * p.heads + h) * p.np;
  const bool load = p.positions[t0] > 0;
  const float m0 = load ? gN[p.dim] : 0.f;
  __syncthreads();
  float m = m0;
  for (int r0 = 0; r0 < p.dim; r0 += blockDim.x) {
    const int r = r0 + threadIdx.x;
    const bool on = r < p.dim;
    float n = load && on ? gN[r] : 0.f;
    m = m0;
    for (int64_t t = t0; t < t1; ++t) {
      const float gi = ml_input_gate(p.z[t * p.z_stride + h], p.cap);
      const float gf = ml_forget_gate(p.z[t * p.z_stride + p.heads + h], p.cap);
      const float m2 = fmaxf(gf + m, gi);
      const float keep = expf(gf + m - m2), add = expf(gi - m2);
      m = m2;
      if (on)
        n = keep * n + add * Elem<T>::load(static_cast<const T*>(p.k) + t * p.in_stride +
                                           h * p.dim + r);
    }
    if (on) gN[r] = n;
  }
  if (threadIdx.x == 0) gN[p.dim] = m;
}

// ------------------------------------------------------------------------ chunked form
// Portion that owns unit u (units cu[i] / ML_UNIT + i .. of portion i); its token range.
struct MlUnit {
  int portion;
  int64_t t0;       // first token
  int count;        // tokens, 0: nobody's unit
  bool first, last; // first / last unit of its portion
};
__device__ __forceinline__ MlUnit ml_unit(const MlstmParams& p, int64_t u) {
  int lo = 0, hi = p.num_portions;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.cu[mid] / ML_UNIT + mid <= u) lo = mid; else hi = mid;
  }
  MlUnit r;
  r.portion = lo;
  const int64_t a = p.cu[lo], b = min((int64_t)p.cu[lo + 1], p.rows);
  const int64_t i = u - (a / ML_UNIT + lo);
  r.t0 = a + i * ML_UNIT;
  const int64_t left = b - r.t0;
  r.count = (int)(left < 0 ? 0 : left > ML_UNIT ? ML_UNIT : left);
  r.first = i == 0;
  r.last = r.t0 + ML_UNIT >= b;
  return r;
}

// CTA = one head of one portion; each warp takes units in turn, some tokens a lane.
constexpr int MG_THREADS = 1024, MG_TPL = ML_UNIT / 32;
constexpr int MG_MAX_UNITS = 4096;            // per portion (524288 tokens)
__global__ void __launch_bounds__(MG_THREADS) mlstm_gates_kernel(const MlstmParams p) {
  extern __shared__ float mg_smem[];          // per unit: sum of f, local maximum, m ahead
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, pi = blockIdx.y;
  const int64_t a = p.cu[pi], b = min((int64_t)p.cu[pi + 1], p.rows);
  if (a < 0 || a >= b) return;
  const int n_units = (int)((b - a + ML_UNIT - 1) / ML_UNIT);
  if (n_units > p.most_units) {               // longer than the caller said
    if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
    return;
  }
  const int64_t u0 = a / ML_UNIT + pi;
  float* tot_f = mg_smem;
  float* tot_m = tot_f + n_units;
  float* m_in = tot_m + n_units;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = MG_THREADS >> 5;
  const int64_t row_of = (int64_t)h * p.units * ML_UNIT;
  for (int u = warp; u < n_units; u += warps) {
    float f[MG_TPL], i[MG_TPL], m[MG_TPL];
#pragma unroll
    for (int e = 0; e < MG_TPL; ++e) {
      const int64_t t = a + (int64_t)u * ML_UNIT + lane * MG_TPL + e;
      const bool on = t < b;
      i[e] = on ? ml_input_gate(p.z[t * p.z_stride + h], p.cap) : ML_NONE;
      f[e] = on ? ml_forget_gate(p.z[t * p.z_stride + p.heads + h], p.cap) : 0.f;
    }
    // (sum of f, maximum of the decayed i) up to and with each token: of this lane's tokens,
    // then over the lanes
    m[0] = i[0];
#pragma unroll
    for (int e = 1; e < MG_TPL; ++e) {
      m[e] = fmaxf(m[e - 1] + f[e], i[e]);
      f[e] += f[e - 1];
    }
    float F = f[MG_TPL - 1], M = m[MG_TPL - 1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, F, o), pm = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) { M = fmaxf(pm + F, M); F += pf; }
    }
    float pf = __shfl_up_sync(0xffffffffu, F, 1), pm = __shfl_up_sync(0xffffffffu, M, 1);
    if (lane == 0) { pf = 0.f; pm = ML_NONE; }
    const int64_t at = row_of + (u0 + u) * ML_UNIT + lane * MG_TPL;
#pragma unroll
    for (int e = 0; e < MG_TPL; ++e) {
      p.gg[at + e] = pf + f[e];
      p.gi[at + e] = i[e];
      p.gm[at + e] = fmaxf(pm + f[e], m[e]);
    }
    if (lane == 31) { tot_f[u] = F; tot_m[u] = M; }
  }
  __syncthreads();
  const int slot = p.slots[a];
  const bool ok = ml_slot_ok(p, slot);
  float* N = p.n_state + ((int64_t)(ok ? slot : 0) * p.heads + h) * p.np;
  if (warp == 0) {
    float m = ok && p.positions[a] > 0 ? N[p.dim] : 0.f;
    for (int v0 = 0; v0 < n_units; v0 += 32) {
      const int u = v0 + lane;
      float F = u < n_units ? tot_f[u] : 0.f, M = u < n_units ? tot_m[u] : ML_NONE;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float pf = __shfl_up_sync(0xffffffffu, F, o), pm = __shfl_up_sync(0xffffffffu, M, o);
        if (lane >= o) { M = fmaxf(pm + F, M); F += pf; }
      }
      const float after = fmaxf(F + m, M);
      float before = __shfl_up_sync(0xffffffffu, after, 1);
      if (lane == 0) before = m;
      if (u < n_units) {
        m_in[u] = before;
        p.unit_m[h * p.units + u0 + u] = before;
        p.unit_decay[h * p.units + u0 + u] = expf(tot_f[u] + before - after);
      }
      m = __shfl_sync(0xffffffffu, after, 31);
    }
    if (ok && lane == 0) N[p.dim] = m;
  }
  __syncthreads();
  for (int u = warp; u < n_units; u += warps) {
    const int64_t at = row_of + (u0 + u) * ML_UNIT + lane * MG_TPL;
#pragma unroll
    for (int e = 0; e < MG_TPL; ++e) p.gm[at + e] = fmaxf(p.gm[at + e], p.gg[at + e] + m_in[u]);
  }
}

// Rows of a unit's q, k or v columns into shared memory [ML_UNIT][pitch], zeros beyond `count`
// rows and `cols` columns up to `cols_p`.
__device__ __forceinline__ void ml_load_rows(const uint16_t* src, int64_t stride, int count,
                                             int cols, int cols_p, uint16_t* dst, int pitch,
                                             bool vec) {
  if (vec) {
    const int packs = cols_p >> 3, total = ML_UNIT * packs;
    constexpr int UN = 8;                      // loads under way
    for (int i0 = threadIdx.x; i0 < total; i0 += UN * blockDim.x) {
      uint4 v[UN];
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int i = i0 + u * blockDim.x, r = i / packs, c = (i - r * packs) * 8;
        v[u] = make_uint4(0u, 0u, 0u, 0u);
        if (i < total && r < count && c < cols)
          v[u] = *reinterpret_cast<const uint4*>(src + r * stride + c);
      }
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int i = i0 + u * blockDim.x, r = i / packs, c = (i - r * packs) * 8;
        if (i < total) *reinterpret_cast<uint4*>(dst + r * pitch + c) = v[u];
      }
    }
  } else {
    for (int i = threadIdx.x; i < ML_UNIT * cols_p; i += blockDim.x) {
      const int r = i / cols_p, c = i - r * cols_p;
      dst[r * pitch + c] = r < count && c < cols ? src[r * stride + c] : (uint16_t)0;
    }
  }
}

// ldmatrix address of a 16 x 16 tile at (row, col) of a [rows][pitch] bf16 array: as an A
// operand (row major), or transposed for arrays that hold the reduction along rows.
__device__ __forceinline__ uint32_t ml_tile(const uint16_t* base, int pitch, int row, int col,
                                            int lane) {
  return smem_u32(base + (row + (lane & 15)) * pitch + col + (lane >> 4) * 8);
}

// acc[8 NT columns] += a (16 x 16) times rows row .. row + 15 of B; the fragments of B come
// ahead of the products.
template <int NT>
__device__ __forceinline__ void ml_products(float (&acc)[NT][4], const uint32_t (&a)[4],
                                            const uint16_t* B, int pitch, int row, int lane) {
  uint32_t b[NT / 2][4];
#pragma unroll
  for (int j = 0; j < NT / 2; ++j)
    ldmatrix_x4_trans(ml_tile(B, pitch, row, j * 16, lane), b[j][0], b[j][1], b[j][2], b[j][3]);
#pragma unroll
  for (int j = 0; j < NT / 2; ++j) {
    mma_bf16_16816(acc[2 * j], a, b[j][0], b[j][1]);
    mma_bf16_16816(acc[2 * j + 1], a, b[j][2], b[j][3]);
  }
}

// CTA = 64 value columns of one head of one unit: inc = sum_s k_s (c_s v_s)^T with
// c_s = e^{g_L - g_s + i_s - m_L}; the CTA of the first columns also sums c_s k_s.
constexpr int MU_THREADS = 256, MU_COLS = 64;
__global__ void __launch_bounds__(MU_THREADS) mlstm_unit_kernel(const MlstmParams p) {
  extern __shared__ uint16_t mu_smem[];        // K [unit][dp + 8] | V hi, lo [unit][72]
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float cs[ML_UNIT];
  const int h = blockIdx.y;
  const int64_t u = blockIdx.z;
  const MlUnit un = ml_unit(p, u);
  if (un.count == 0) return;
  const int dp = (p.dim + 15) & ~15, kp = dp + 8, vpit = MU_COLS + 8;
  uint16_t* K = mu_smem;
  uint16_t* Vh = K + ML_UNIT * kp;
  uint16_t* Vl = Vh + ML_UNIT * vpit;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int v0 = blockIdx.x * MU_COLS;
  const uint16_t* kg = static_cast<const uint16_t*>(p.k) + un.t0 * p.in_stride + h * p.dim;
  const uint16_t* vg = static_cast<const uint16_t*>(p.v) + un.t0 * p.in_stride + h * p.vdim + v0;
  // this thread's pieces of v come while the others are brought in
  constexpr int VN = ML_UNIT * (MU_COLS / 8) / MU_THREADS;
  const int cols = min(MU_COLS, p.vdim - v0);
  uint4 vx[VN];
#pragma unroll
  for (int j = 0; j < VN; ++j) {
    const int i = tid + j * MU_THREADS, r = i / (MU_COLS / 8), c = (i % (MU_COLS / 8)) * 8;
    vx[j] = make_uint4(0u, 0u, 0u, 0u);
    if (r < un.count && c < cols) {
      if (p.vdim % 8 == 0) {
        vx[j] = *reinterpret_cast<const uint4*>(vg + r * p.in_stride + c);
      } else {
        uint16_t e[8];
#pragma unroll
        for (int x = 0; x < 8; ++x) e[x] = c + x < cols ? vg[r * p.in_stride + c + x] : (uint16_t)0;
        vx[j] = make_uint4(e[0] | (uint32_t)e[1] << 16, e[2] | (uint32_t)e[3] << 16,
                           e[4] | (uint32_t)e[5] << 16, e[6] | (uint32_t)e[7] << 16);
      }
    }
  }
  const int64_t at = (int64_t)h * p.units * ML_UNIT + u * ML_UNIT;
  if (tid < ML_UNIT)
    cs[tid] = expf(p.gg[at + ML_UNIT - 1] - p.gg[at + tid] + p.gi[at + tid] -
                   p.gm[at + ML_UNIT - 1]);
  ml_load_rows(kg, p.in_stride, un.count, p.dim, dp, K, kp, p.dim % 8 == 0);
  __syncthreads();
#pragma unroll
  for (int j = 0; j < VN; ++j) {
    const int i = tid + j * MU_THREADS, r = i / (MU_COLS / 8), c = (i % (MU_COLS / 8)) * 8;
    const float k = cs[r];
    const uint4 x = vx[j];
    uint4 hi, lo;
    split_bf16(bf16lo(x.x) * k, bf16hi(x.x) * k, &hi.x, &lo.x);
    split_bf16(bf16lo(x.y) * k, bf16hi(x.y) * k, &hi.y, &lo.y);
    split_bf16(bf16lo(x.z) * k, bf16hi(x.z) * k, &hi.z, &lo.z);
    split_bf16(bf16lo(x.w) * k, bf16hi(x.w) * k, &hi.w, &lo.w);
    *reinterpret_cast<uint4*>(Vh + r * vpit + c) = hi;
    *reinterpret_cast<uint4*>(Vl + r * vpit + c) = lo;
  }
  __syncthreads();
  float* inc = p.inc + (u * p.heads + h) * p.dim * p.vp;
  if (blockIdx.x == 0)
    for (int r = tid; r < p.dim; r += MU_THREADS) {
      float s = 0.f;                              // rows beyond the count are zeros
#pragma unroll 16
      for (int t = 0; t < ML_UNIT; ++t) s = fmaf(cs[t], bf16_bits_to_float(K[t * kp + r]), s);
      p.ninc[(u * p.heads + h) * p.dim + r] = s;
    }
  const int gr = lane >> 2, tq = lane & 3;
  for (int d0 = warp * 16; d0 < dp; d0 += MU_THREADS / 32 * 16) {
    float acc[8][4] = {};
#pragma unroll
    for (int ks = 0; ks < ML_UNIT; ks += 16) {
      // A = K^T: rows are key channels, the reduction runs over tokens
      uint32_t a[4];
      ldmatrix_x4_trans(smem_u32(K + (ks + (lane & 7) + (lane >> 4) * 8) * kp + d0 +
                                 ((lane >> 3) & 1) * 8), a[0], a[1], a[2], a[3]);
      ml_products<8>(acc, a, Vh, vpit, ks, lane);
      ml_products<8>(acc, a, Vl, vpit, ks, lane);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = d0 + gr + e * 8, c = v0 + j * 8 + tq * 2;
        if (r < p.dim && c < p.vp)              // vp is even; columns beyond vdim are zeros
          *reinterpret_cast<float2*>(inc + (int64_t)r * p.vp + c) =
              make_float2(acc[j][e * 2], acc[j][e * 2 + 1]);
      }
  }
}

// Thread = four elements of S (or one of n) of one head of one portion: the value ahead of
// every unit replaces what the unit adds, S as (high, low) bf16 pairs.
__global__ void __launch_bounds__(256) mlstm_carry_kernel(const MlstmParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, pi = blockIdx.z;
  const int64_t a = p.cu[pi], b = min((int64_t)p.cu[pi + 1], p.rows);
  if (a < 0 || a >= b) return;
  const int n_units = (int)((b - a + ML_UNIT - 1) / ML_UNIT);
  const int64_t u0 = a / ML_UNIT + pi;
  const int slot = p.slots[a];
  const bool ok = ml_slot_ok(p, slot);
  const bool load = ok && p.positions[a] > 0;
  const float* dec = p.unit_decay + h * p.units + u0;
  const int quads = p.dim * (p.vp >> 2);
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  const int64_t at = (int64_t)(ok ? slot : 0) * p.heads + h;
  if (i < quads) {
    float4* st = reinterpret_cast<float4*>(p.s_state + at * p.dim * p.vp) + i;
    float4 s = load ? *st : make_float4(0.f, 0.f, 0.f, 0.f);
    const int64_t step = (int64_t)p.heads * quads;
    float4* inc = reinterpret_cast<float4*>(p.inc) + (u0 * p.heads + h) * quads + i;
    constexpr int UN = 4;
    for (int u = 0; u < n_units; u += UN) {
      float4 d[UN];
      float k[UN];
#pragma unroll
      for (int e = 0; e < UN; ++e)
        if (u + e < n_units) {
          d[e] = inc[(u + e) * step];
          k[e] = dec[u + e];
        }
#pragma unroll
      for (int e = 0; e < UN; ++e)
        if (u + e < n_units) {
          uint32_t h0, l0, h1, l1;
          split_bf16(s.x, s.y, &h0, &l0);
          split_bf16(s.z, s.w, &h1, &l1);
          *reinterpret_cast<uint4*>(inc + (u + e) * step) = make_uint4(h0, h1, l0, l1);
          s = s * k[e] + d[e];
        }
    }
    if (ok) *st = s;
    return;
  }
  const int r = i - quads;
  if (r >= p.dim) return;
  float* st = p.n_state + at * p.np + r;
  float s = load ? *st : 0.f;
  for (int u = 0; u < n_units; ++u) {
    float* q = p.ninc + ((u0 + u) * p.heads + h) * p.dim + r;
    const float d = *q;
    *q = s;
    s = s * dec[u] + d;
  }
  if (ok) *st = s;
}

// CTA = one head of one unit, 16 tokens a warp.  Value columns go 32 at a time.
constexpr int MO_THREADS = ML_UNIT / 16 * 32, MO_COLS = 32, MO_KT = ML_UNIT / 16;
__host__ __device__ constexpr int mo_smem(int dp) {
  return (2 * ML_UNIT * (dp + 8) + ML_UNIT * (MO_COLS + 8) + 2 * dp * (MO_COLS + 8)) * 2 +
         (3 * ML_UNIT + dp) * 4;
}
__global__ void __launch_bounds__(MO_THREADS, 2) mlstm_output_kernel(const MlstmParams p) {
  extern __shared__ uint16_t mo_raw[];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x;
  const int64_t u = blockIdx.y;
  const MlUnit un = ml_unit(p, u);
  if (un.count == 0) return;
  const int dp = (p.dim + 15) & ~15, kp = dp + 8, vpit = MO_COLS + 8;
  uint16_t* Q = mo_raw;
  uint16_t* K = Q + ML_UNIT * kp;
  uint16_t* V = K + ML_UNIT * kp;
  uint16_t* Sh = V + ML_UNIT * vpit;
  uint16_t* Sl = Sh + dp * vpit;
  float* g = reinterpret_cast<float*>(Sl + dp * vpit);   // g | i - g | m | n
  float* ig = g + ML_UNIT;
  float* ms = ig + ML_UNIT;
  float* n = ms + ML_UNIT;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gr = lane >> 2, tq = lane & 3;
  const uint16_t* qg = static_cast<const uint16_t*>(p.q) + un.t0 * p.in_stride + h * p.dim;
  const uint16_t* kg = static_cast<const uint16_t*>(p.k) + un.t0 * p.in_stride + h * p.dim;
  const uint16_t* vg = static_cast<const uint16_t*>(p.v) + un.t0 * p.in_stride + h * p.vdim;
  ml_load_rows(qg, p.in_stride, un.count, p.dim, dp, Q, kp, p.dim % 8 == 0);
  ml_load_rows(kg, p.in_stride, un.count, p.dim, dp, K, kp, p.dim % 8 == 0);
  const int64_t at = (int64_t)h * p.units * ML_UNIT + u * ML_UNIT;
  if (tid < ML_UNIT) {
    const float gt = p.gg[at + tid];
    g[tid] = gt;
    ig[tid] = p.gi[at + tid] - gt;
    ms[tid] = p.gm[at + tid];
  }
  for (int r = tid; r < dp; r += MO_THREADS)
    n[r] = r < p.dim ? p.ninc[(u * p.heads + h) * p.dim + r] : 0.f;
  const float m_in = p.unit_m[h * p.units + u];
  __syncthreads();
  // scores of this warp's 16 tokens against the unit's tokens up to them, decayed
  const int r0 = warp * 16;
  const float g0 = g[r0 + gr], g1 = g[r0 + gr + 8], m0 = ms[r0 + gr], m1 = ms[r0 + gr + 8];
  uint32_t ph[MO_KT][4], pl[MO_KT][4];          // A fragments of the decayed scores
  float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
  for (int kt = 0; kt < MO_KT; ++kt) {
#pragma unroll
    for (int i = 0; i < 4; ++i) ph[kt][i] = pl[kt][i] = 0u;
    if (kt > warp) continue;
    float s[2][4] = {};
    for (int d = 0; d < dp; d += 16) {
      uint32_t a[4], b[4];
      ldmatrix_x4(ml_tile(Q, kp, r0, d, lane), a[0], a[1], a[2], a[3]);
      // 16 keys x 16 channels, keys along n
      ldmatrix_x4(smem_u32(K + (kt * 16 + (lane & 7) + (lane >> 4) * 8) * kp + d +
                           ((lane >> 3) & 1) * 8), b[0], b[1], b[2], b[3]);
      mma_bf16_16816(s[0], a, b[0], b[1]);
      mma_bf16_16816(s[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = kt * 16 + j * 8 + tq * 2 + e;
        const float x = ig[c];
        s[j][e] = c <= r0 + gr ? s[j][e] * p.q_scale * __expf(g0 + x - m0) : 0.f;
        s[j][2 + e] = c <= r0 + gr + 8 ? s[j][2 + e] * p.q_scale * __expf(g1 + x - m1) : 0.f;
        sum0 += s[j][e];
        sum1 += s[j][2 + e];
      }
    split_bf16(s[0][0], s[0][1], &ph[kt][0], &pl[kt][0]);
    split_bf16(s[0][2], s[0][3], &ph[kt][1], &pl[kt][1]);
    split_bf16(s[1][0], s[1][1], &ph[kt][2], &pl[kt][2]);
    split_bf16(s[1][2], s[1][3], &ph[kt][3], &pl[kt][3]);
  }
  float qn0 = 0.f, qn1 = 0.f;
  for (int d = tq; d < dp; d += 4) {
    qn0 = fmaf(bf16_bits_to_float(Q[(r0 + gr) * kp + d]), n[d], qn0);
    qn1 = fmaf(bf16_bits_to_float(Q[(r0 + gr + 8) * kp + d]), n[d], qn1);
  }
  const float in0 = expf(g0 + m_in - m0) * p.q_scale, in1 = expf(g1 + m_in - m1) * p.q_scale;
  sum0 += in0 * qn0;
  sum1 += in1 * qn1;
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, o);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, o);
  }
  const float inv0 = 1.0f / (fmaxf(fabsf(sum0), expf(-m0)) + ML_EPS);
  const float inv1 = 1.0f / (fmaxf(fabsf(sum1), expf(-m1)) + ML_EPS);
  const int64_t hv = (int64_t)p.heads * p.vdim;
  const uint2* st = reinterpret_cast<const uint2*>(p.inc + (u * p.heads + h) * p.dim * p.vp);
  for (int v0 = 0; v0 < p.vdim; v0 += MO_COLS) {
    const int cols = min(MO_COLS, p.vdim - v0);
    __syncthreads();
    ml_load_rows(vg + v0, p.in_stride, un.count, cols, MO_COLS, V, vpit,
                 p.vdim % 8 == 0);
    constexpr int SN = 4;                      // loads under way
    for (int i0 = tid; i0 < dp * (MO_COLS / 4); i0 += SN * MO_THREADS) {
      uint4 x[SN];
#pragma unroll
      for (int j = 0; j < SN; ++j) {
        const int i = i0 + j * MO_THREADS, r = i / (MO_COLS / 4), c = (i % (MO_COLS / 4)) * 4;
        x[j] = make_uint4(0u, 0u, 0u, 0u);
        if (r < p.dim && v0 + c < p.vp)
          x[j] = *reinterpret_cast<const uint4*>(st + ((int64_t)r * p.vp + v0 + c) / 2);
      }
#pragma unroll
      for (int j = 0; j < SN; ++j) {
        const int i = i0 + j * MO_THREADS, r = i / (MO_COLS / 4), c = (i % (MO_COLS / 4)) * 4;
        if (r >= dp) continue;
        *reinterpret_cast<uint2*>(Sh + r * vpit + c) = make_uint2(x[j].x, x[j].y);
        *reinterpret_cast<uint2*>(Sl + r * vpit + c) = make_uint2(x[j].z, x[j].w);
      }
    }
    __syncthreads();
    constexpr int NT = MO_COLS / 8;
    float acc[NT][4] = {};
    for (int d = 0; d < dp; d += 16) {
      uint32_t a[4];
      ldmatrix_x4(ml_tile(Q, kp, r0, d, lane), a[0], a[1], a[2], a[3]);
      ml_products<NT>(acc, a, Sh, vpit, d, lane);
      ml_products<NT>(acc, a, Sl, vpit, d, lane);
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][0] *= in0; acc[j][1] *= in0;
      acc[j][2] *= in1; acc[j][3] *= in1;
    }
#pragma unroll
    for (int kt = 0; kt < MO_KT; ++kt) {
      if (kt > warp) continue;
      ml_products<NT>(acc, ph[kt], V, vpit, kt * 16, lane);
      ml_products<NT>(acc, pl[kt], V, vpit, kt * 16, lane);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = r0 + gr + e * 8;
      if (r >= un.count) continue;
      float* o = p.o + (un.t0 + r) * hv + h * p.vdim + v0;
      const float inv = e ? inv1 : inv0;
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int c = j * 8 + tq * 2;
        if (c + 1 < cols && (p.vdim & 1) == 0) {
          *reinterpret_cast<float2*>(o + c) =
              make_float2(acc[j][e * 2] * inv, acc[j][e * 2 + 1] * inv);
        } else {
          if (c < cols) o[c] = acc[j][e * 2] * inv;
          if (c + 1 < cols) o[c + 1] = acc[j][e * 2 + 1] * inv;
        }
      }
    }
  }
}

static int64_t ml_units(int64_t rows, int portions) { return rows / ML_UNIT + portions; }

static int ml_check(const MlstmParams& p, const char* who) {
  FK_REQUIRE(p.rows >= 0 && p.heads > 0 && p.dim > 0 && p.vdim > 0 && p.num_slots > 0 &&
                 p.cap > 0.f,
             FK_ERR_INVALID_ARG, "%s: bad sizes", who);
  FK_REQUIRE(p.q && p.k && p.v && p.z && p.s_state && p.n_state && p.slots && p.positions,
             FK_ERR_INVALID_ARG, "%s: null pointer", who);
  FK_REQUIRE(p.vdim <= 1024 && p.dim <= 512, FK_ERR_UNSUPPORTED, "%s: head size %d x %d too large",
             who, p.dim, p.vdim);
  FK_REQUIRE(p.z_stride >= 2 * p.heads, FK_ERR_INVALID_ARG, "%s: bad stride", who);
  FK_REQUIRE(aligned16(p.s_state) && aligned16(p.n_state) && aligned16(p.q) && aligned16(p.k) &&
                 aligned16(p.v) && p.in_stride % 8 == 0,
             FK_ERR_ALIGNMENT, "%s: operands must be 16-byte aligned", who);
  return FK_OK;
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_mlstm_state_cols(int vdim) { return (vdim + 3) / 4 * 4; }
int fk_mlstm_norm_cols(int dim) { return (dim + 1 + 3) / 4 * 4; }

int fk_mlstm_step(const void* q, const void* k, const void* v, int64_t in_stride, int is_f32,
                  const float* z, int64_t z_stride, const void* gate, int64_t gate_stride,
                  const float* weight, float* s_state, float* n_state, int num_slots,
                  const int32_t* slots, const int64_t* positions, void* out, int64_t out_stride,
                  int64_t rows, int heads, int dim, int vdim, float gate_cap, float q_scale,
                  float eps, int32_t* status, fk_stream_t stream) {
  MlstmParams p{};
  p.q = q; p.k = k; p.v = v; p.in_stride = in_stride; p.z = z; p.z_stride = z_stride;
  p.gate = gate; p.gate_stride = gate_stride; p.weight = weight; p.s_state = s_state;
  p.n_state = n_state; p.num_slots = num_slots; p.slots = slots; p.positions = positions;
  p.out = out; p.out_stride = out_stride; p.rows = rows; p.heads = heads; p.dim = dim;
  p.vdim = vdim; p.vp = fk_mlstm_state_cols(vdim); p.np = fk_mlstm_norm_cols(dim);
  p.cap = gate_cap; p.q_scale = q_scale; p.eps = eps; p.status = status;
  if (rows == 0) return FK_OK;
  const int rc = ml_check(p, "fk_mlstm_step");
  if (rc != FK_OK) return rc;
  FK_REQUIRE(gate && weight && out, FK_ERR_INVALID_ARG, "fk_mlstm_step: null pointer");
  FK_REQUIRE(out_stride >= (int64_t)heads * vdim && gate_stride >= (int64_t)heads * vdim,
             FK_ERR_INVALID_ARG, "fk_mlstm_step: bad stride");
  FK_REQUIRE(rows <= 65535, FK_ERR_UNSUPPORTED, "fk_mlstm_step: too many rows");
  const int groups = MS_THREADS / (p.vp / 4);
  const size_t smem = ((size_t)2 * ((dim + 3) & ~3) + (size_t)groups * p.vp) * 4;
  const dim3 grid((unsigned)heads, (unsigned)rows);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32 ? launch_kernel(mlstm_step_kernel<float>, grid, dim3(MS_THREADS), smem, s, p)
                    : launch_kernel(mlstm_step_kernel<uint16_t>, grid, dim3(MS_THREADS), smem, s,
                                    p));
  count_launch();
  return FK_OK;
}

int64_t fk_mlstm_workspace_floats(int64_t rows, int num_portions, int heads, int dim, int vdim) {
  const int64_t units = ml_units(rows, num_portions);
  const int64_t vp = fk_mlstm_state_cols(vdim);
  const int64_t gates = 3 * heads * units * ML_UNIT + ((2 * heads * units + 3) & ~3ll);
  return gates + units * heads * dim * (vp + 1);
}

int fk_mlstm_portions(const void* q, const void* k, const void* v, int64_t in_stride, int is_f32,
                      const float* z, int64_t z_stride, float* s_state, float* n_state,
                      int num_slots, const int32_t* cu_portions, int num_portions,
                      const int32_t* slots, const int64_t* positions, float* o, int64_t rows,
                      int heads, int dim, int vdim, float gate_cap, float q_scale,
                      float* workspace, int64_t workspace_floats, int64_t longest,
                      int32_t* status, fk_stream_t stream) {
  MlstmParams p{};
  p.q = q; p.k = k; p.v = v; p.in_stride = in_stride; p.z = z; p.z_stride = z_stride;
  p.s_state = s_state; p.n_state = n_state; p.num_slots = num_slots; p.cu = cu_portions;
  p.num_portions = num_portions; p.slots = slots; p.positions = positions; p.o = o;
  p.rows = rows; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.vp = fk_mlstm_state_cols(vdim); p.np = fk_mlstm_norm_cols(dim); p.cap = gate_cap;
  p.q_scale = q_scale; p.status = status;
  if (rows == 0 || num_portions == 0) return FK_OK;
  int rc = ml_check(p, "fk_mlstm_portions");
  if (rc != FK_OK) return rc;
  FK_REQUIRE(cu_portions && o && num_portions > 0, FK_ERR_INVALID_ARG,
             "fk_mlstm_portions: null pointer");
  FK_REQUIRE(num_portions <= 65535 && heads <= 65535, FK_ERR_UNSUPPORTED,
             "fk_mlstm_portions: too many portions or heads");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int64_t units = ml_units(rows, num_portions);
  const bool chunked = !is_f32 && workspace != nullptr && dim <= 256 && units <= 65535 &&
                       longest <= (int64_t)MG_MAX_UNITS * ML_UNIT;
  if (!chunked) {
    const size_t smem = (size_t)dim * (MC_COLS + 5) * 4;
    const dim3 grid((unsigned)((vdim + MC_COLS - 1) / MC_COLS), (unsigned)heads,
                    (unsigned)num_portions);
    const dim3 ngrid((unsigned)heads, (unsigned)num_portions);
    static PerDeviceOnce once_f, once_h;
    FK_CUDA_OK(set_max_dynamic_smem(once_f, mlstm_scan_kernel<float>, 512 * (MC_COLS + 5) * 4));
    FK_CUDA_OK(set_max_dynamic_smem(once_h, mlstm_scan_kernel<uint16_t>, 512 * (MC_COLS + 5) * 4));
    if (is_f32) {
      FK_CUDA_OK(launch_kernel(mlstm_scan_kernel<float>, grid, dim3(MC_COLS * MC_GROUPS), smem, s,
                               p));
      FK_CUDA_OK(launch_kernel(mlstm_scan_norm_kernel<float>, ngrid, dim3(128), 0, s, p));
    } else {
      FK_CUDA_OK(launch_kernel(mlstm_scan_kernel<uint16_t>, grid, dim3(MC_COLS * MC_GROUPS), smem,
                               s, p));
      FK_CUDA_OK(launch_kernel(mlstm_scan_norm_kernel<uint16_t>, ngrid, dim3(128), 0, s, p));
    }
    count_launch(2);
    return FK_OK;
  }
  FK_REQUIRE(aligned16(workspace) && workspace_floats >= fk_mlstm_workspace_floats(
                 rows, num_portions, heads, dim, vdim),
             FK_ERR_WORKSPACE, "fk_mlstm_portions: workspace too small");
  p.units = units;
  const int64_t per = (int64_t)heads * units * ML_UNIT;
  p.gg = workspace; p.gi = p.gg + per; p.gm = p.gi + per;
  p.unit_m = p.gm + per; p.unit_decay = p.unit_m + heads * units;
  p.inc = workspace + 3 * per + ((2 * heads * units + 3) & ~3ll);
  p.ninc = p.inc + units * heads * dim * p.vp;
  const int64_t most_units = (longest + ML_UNIT - 1) / ML_UNIT;
  p.most_units = (int)most_units;
  static PerDeviceOnce once_g, once_u, once_o;
  FK_CUDA_OK(set_max_dynamic_smem(once_g, mlstm_gates_kernel, MG_MAX_UNITS * 3 * 4));
  const dim3 pg((unsigned)heads, (unsigned)num_portions);
  FK_CUDA_OK(launch_kernel(mlstm_gates_kernel, pg, dim3(MG_THREADS), (size_t)most_units * 3 * 4, s,
                           p));
  const int dp = (dim + 15) & ~15;
  const int usmem = (ML_UNIT * (dp + 8) + 2 * ML_UNIT * (MU_COLS + 8)) * 2;
  FK_CUDA_OK(set_max_dynamic_smem(once_u, mlstm_unit_kernel,
                                  (ML_UNIT * (256 + 8) + 2 * ML_UNIT * (MU_COLS + 8)) * 2));
  const dim3 ug((unsigned)((vdim + MU_COLS - 1) / MU_COLS), (unsigned)heads, (unsigned)units);
  FK_CUDA_OK(launch_kernel(mlstm_unit_kernel, ug, dim3(MU_THREADS), (size_t)usmem, s, p));
  const int64_t work = (int64_t)dim * (p.vp / 4) + dim;
  const dim3 cg((unsigned)((work + 255) / 256), (unsigned)heads, (unsigned)num_portions);
  FK_CUDA_OK(launch_kernel(mlstm_carry_kernel, cg, dim3(256), 0, s, p));
  FK_CUDA_OK(set_max_dynamic_smem(once_o, mlstm_output_kernel, mo_smem(256)));
  const dim3 og((unsigned)heads, (unsigned)units);
  FK_CUDA_OK(launch_kernel(mlstm_output_kernel, og, dim3(MO_THREADS), (size_t)mo_smem(dp), s, p));
  count_launch(4);
  return FK_OK;
}

}  // extern "C"
