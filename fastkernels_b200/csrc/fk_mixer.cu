// Row kernels around sublayers with an fp32 residual stream, for bf16 and fp32
// activations:
//
//   fk_embed_f32            residual row = embedding row
//   fk_norm_shift           add the normed sublayer output, norm with ONE gain, token
//                           shift against the previous token (kept per sequence)
//   fk_branch_combine       normed half-sum of two mixers' outputs -> residual -> norm
//   fk_rope_rms_store       interleaved partial RoPE + weight-less per-head RMS norm of
//                           q and k, store of k and of the raw projection as value
//   fk_act_and_mul          act(gate) * up, SiLU or tanh-GELU
//
// All of them are bound by HBM traffic; rows are padded to a multiple of 64
// elements whose tail is zero, so every access is a full 8- or 16-byte vector.
// Norms, angles, the residual and the shifted row are fp32 until the one rounding
// to the activation type at the end.
#include "fk_types.cuh"

namespace fk {

constexpr int MX_MAX_VPT = 4;   // float4 groups of a row per thread

// One row as registers: group i of thread t is float4 number t + i * blockDim.
template <int VPT>
struct Row {
  float4 v[VPT];
};

struct NormShiftParams {
  const float* x_in; float* x_out;       // [T, stride]
  const void* y;                         // sublayer output [T, y_stride] or null
  const float* y_gain;                   // its norm's gain
  const float* gain;                     // gain of the norm that feeds the next sublayer
  const float* shift;                    // [stride] or null: no token shift
  void* out;                             // [T, stride]
  float* state;                          // [slots, stride]: previous normed row
  const int32_t* slots;                  // [T] state slot of a token, -1: none
  const int64_t* positions;              // [T]
  const int32_t* cu; int num_portions;   // token ranges of the portions
  int64_t rows, y_stride; int stride, width; int num_slots;
  float eps; int rows_per_cta;
  int32_t* status;
};

// The loads of one row.
template <typename T, int VPT>
__device__ __forceinline__ void load_row(const NormShiftParams& p, int64_t t, Row<VPT>& x,
                                         Row<VPT>& y) {
  const int groups = p.stride >> 2;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int g = threadIdx.x + i * blockDim.x;
    x.v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    y.v[i] = x.v[i];
    if (g < groups) {
      x.v[i] = *reinterpret_cast<const float4*>(p.x_in + t * p.stride + g * 4);
      if (p.y) y.v[i] = Elem<T>::load4(static_cast<const T*>(p.y) + t * p.y_stride + g * 4);
    }
  }
}

// x' = x + rms(y) * y_gain, stored when asked; h (in: x) = rms(x') * gain.
//
// One reduction for both norms: with c = rms scale of y times its gain,
// sum x'^2 = sum x^2 + 2 c sum x y + c^2 sum y^2.  Where x and c y cancel to less than a
// hundredth that would lose digits, and sum x'^2 is taken from x' itself.
template <typename T, int VPT>
__device__ __forceinline__ void norm_row(const NormShiftParams& p, int64_t t, bool store_x,
                                         Row<VPT>& h, const Row<VPT>& y, float* red, int& flip) {
  const int groups = p.stride >> 2;
  const float inv_w = 1.0f / (float)p.width;
  float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    s[0] += sumsq(h.v[i]);
    if (p.y) {
      const float4 xy = h.v[i] * y.v[i];
      s[1] += (xy.x + xy.y) + (xy.z + xy.w);
      s[2] += sumsq(y.v[i]);
    }
  }
  block_sums<3>(s, red, flip);
  float ss = s[0];
  if (p.y) {
    const float c = rsqrtf(s[2] * inv_w + p.eps) * *p.y_gain;
#pragma unroll
    for (int i = 0; i < VPT; ++i) h.v[i] = h.v[i] + y.v[i] * c;
    const float all = s[0] + c * c * s[2];
    ss = all + 2.0f * c * s[1];
    if (ss < 0.01f * all) {
      float e[3] = {0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < VPT; ++i) e[0] += sumsq(h.v[i]);
      block_sums<3>(e, red, flip);
      ss = e[0];
    }
  }
  if (store_x && p.x_out) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int g = threadIdx.x + i * blockDim.x;
      if (g < groups) *reinterpret_cast<float4*>(p.x_out + t * p.stride + g * 4) = h.v[i];
    }
  }
  const float sc = rsqrtf(ss * inv_w + p.eps) * *p.gain;
#pragma unroll
  for (int i = 0; i < VPT; ++i) h.v[i] = h.v[i] * sc;
}

// A CTA walks `rows_per_cta` consecutive rows and carries the normed row from one to
// the next.  The row ahead of its first one is computed once more (from x_in, which this
// kernel does not change), or comes from the sequence's state when a portion starts
// there.  The state of a portion is read AND replaced by the CTA that owns the portion's
// first row (for that it computes the portion's last row, if it is not one of its own),
// so no other CTA touches it.
template <typename T, int VPT, bool SHIFT>
__global__ void __launch_bounds__(512, VPT == 1 ? 4 : VPT == 2 ? 3 : VPT == 4 ? 2 : 1)
norm_shift_kernel(const NormShiftParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[192];
  int flip = 0;
  const int groups = p.stride >> 2;
  const int64_t t0 = (int64_t)blockIdx.x * p.rows_per_cta;
  const int n = (int)min((int64_t)p.rows_per_cta, p.rows - t0);
  // the previous normed row: a thread only ever touches its own entries
  __shared__ float4 prev[SHIFT ? VPT * 512 : 1];
  float* pend = nullptr;        // state that waits for row pend_row
  int64_t pend_row = -1;
  int it = 0;
  if (SHIFT && t0 > 0) {
    const int slot = p.slots[t0];
    if (slot >= 0 && p.slots[t0 - 1] == slot) it = -1;
  }
  for (; it < n || (SHIFT && pend != nullptr); ++it) {
    const bool own = it >= 0 && it < n;
    const int64_t t = it < n ? t0 + it : pend_row;
    Row<VPT> h, y;
    load_row<T, VPT>(p, t, h, y);
    if (SHIFT && own) {
      const int slot = p.slots[t];
      if (slot < 0 || t == 0 || p.slots[t - 1] != slot) {
        const bool in_range = slot >= 0 && slot < p.num_slots;
        if (slot >= p.num_slots && threadIdx.x == 0 && p.status)
          atomicOr(p.status, FK_DEV_BAD_SLOT);
        const bool from_state = in_range && p.positions[t] > 0;
        float* st = p.state + (int64_t)(in_range ? slot : 0) * p.stride;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int g = threadIdx.x + i * blockDim.x;
          if (g < groups)
            prev[g] = from_state ? *reinterpret_cast<const float4*>(st + g * 4)
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        pend = nullptr;
        if (in_range) {
          // last row of the portion that starts here
          int lo = 0, hi = p.num_portions;
          while (hi - lo > 1) {
            const int mid = (lo + hi) >> 1;
            if (p.cu[mid] <= t) lo = mid; else hi = mid;
          }
          pend = st;
          pend_row = max(t, min((int64_t)p.cu[lo + 1], p.rows) - 1);
        }
      }
    }
    norm_row<T, VPT>(p, t, own, h, y, red, flip);
    if (SHIFT && pend != nullptr && t == pend_row) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int g = threadIdx.x + i * blockDim.x;
        if (g < groups) *reinterpret_cast<float4*>(pend + g * 4) = h.v[i];
      }
      pend = nullptr;
    }
    if (own) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int g = threadIdx.x + i * blockDim.x;
        if (g < groups) {
          float4 o = h.v[i];
          if (SHIFT) {
            const float4 sh = __ldg(reinterpret_cast<const float4*>(p.shift + g * 4));
            o = o + (prev[g] - o) * sh;
          }
          Elem<T>::store4(static_cast<T*>(p.out) + t * p.stride + g * 4, o);
        }
      }
    }
    if (SHIFT) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int g = threadIdx.x + i * blockDim.x;
        if (g < groups) prev[g] = h.v[i];
      }
    }
  }
}

struct CombineParams {
  const void* a; const void* b;          // [T, ab_stride] outputs of the two mixers
  const float* wa; const float* wb;      // [stride] norm weights
  const float* gain_out;                 // gain of the norm after the mixer
  const float* gain;                     // gain of the norm ahead of the feed-forward
  float* x;                              // residual [T, stride], in place
  void* out;                             // [T, stride] or null
  int64_t rows, ab_stride; int stride, width;
  float eps;
};

template <typename T, int VPT>
__global__ void __launch_bounds__(512) branch_combine_kernel(const CombineParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[128];
  int flip = 0;
  const int groups = p.stride >> 2;
  const float inv_w = 1.0f / (float)p.width;
  const int64_t t = blockIdx.x;
  float4 a[VPT], b[VPT], x[VPT];
  float s2[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int g = threadIdx.x + i * blockDim.x;
    a[i] = b[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (g < groups) {
      a[i] = Elem<T>::load4(static_cast<const T*>(p.a) + t * p.ab_stride + g * 4);
      b[i] = Elem<T>::load4(static_cast<const T*>(p.b) + t * p.ab_stride + g * 4);
      x[i] = *reinterpret_cast<const float4*>(p.x + t * p.stride + g * 4);
    }
    s2[0] += sumsq(a[i]);
    s2[1] += sumsq(b[i]);
  }
  block_sums<2>(s2, red, flip);
  const float ra = 0.5f * rsqrtf(s2[0] * inv_w + p.eps);
  const float rb = 0.5f * rsqrtf(s2[1] * inv_w + p.eps);
  float s[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int g = threadIdx.x + i * blockDim.x;
    if (g < groups) {
      const float4 wa = __ldg(reinterpret_cast<const float4*>(p.wa + g * 4));
      const float4 wb = __ldg(reinterpret_cast<const float4*>(p.wb + g * 4));
      a[i] = (a[i] * ra) * wa + (b[i] * rb) * wb;
    }
    s[0] += sumsq(a[i]);
  }
  // the two reductions alternate between the halves of `red`: the first used
  // floats 0..63 (two values per warp), this one starts at 64
  float* red1 = red + 64;
  int flip1 = 0;
  block_sums<1>(s, red1, flip1);
  const float rm = rsqrtf(s[0] * inv_w + p.eps) * *p.gain_out;
  float sx[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int g = threadIdx.x + i * blockDim.x;
    x[i] = x[i] + a[i] * rm;
    if (g < groups) *reinterpret_cast<float4*>(p.x + t * p.stride + g * 4) = x[i];
    sx[0] += sumsq(x[i]);
  }
  if (!p.out) return;
  block_sums<1>(sx, red1, flip1);
  const float rx = rsqrtf(sx[0] * inv_w + p.eps) * *p.gain;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int g = threadIdx.x + i * blockDim.x;
    if (g < groups) Elem<T>::store4(static_cast<T*>(p.out) + t * p.stride + g * 4, x[i] * rx);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) embed_f32_kernel(
    const T* __restrict__ table, const int64_t* __restrict__ ids, float* __restrict__ x,
    int64_t rows, int groups, int64_t vocab, int32_t* status) {
  pdl_launch_dependents();
  pdl_wait();
  for (int64_t t = blockIdx.x; t < rows; t += gridDim.x) {
    const int64_t id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0 && status) atomicOr(status, FK_DEV_BAD_SLOT);
    for (int g = threadIdx.x; g < groups; g += blockDim.x) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (ok) v = Elem<T>::load4(table + (id * groups + g) * 4);
      *reinterpret_cast<float4*>(x + (t * groups + g) * 4) = v;
    }
  }
}

struct RopeRmsParams {
  const void* q; const void* k; int64_t in_stride;   // [T, in_stride] packed projection rows
  void* q_out;                                       // [T, hkv * gp, dp]
  void* k_cache; void* v_cache;                      // [slots, hkv, dp]
  const int64_t* positions; const int32_t* slots;
  const float* cos_sin; int64_t max_position;        // [max_position, rot] = cos | sin
  int64_t rows, num_slots;
  int hkv, g, gp, d, dp, rot;
  float eps;
  int32_t* status;
};

// One warp per (token, head).  Pair e of a head is (2e, 2e + 1); pairs below rot / 2
// are rotated, the rest pass.  A head's slots beyond d are written as zeros, and so
// are whole query heads beyond a group's own.
template <typename T, int PPL>
__global__ void __launch_bounds__(256) rope_rms_store_kernel(const RopeRmsParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int qheads = p.hkv * p.gp;
  const int heads = qheads + p.hkv;
  const int h = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (h >= heads) return;
  const bool is_q = h < qheads;
  const int kvh = is_q ? h / p.gp : h - qheads;
  const int in_group = is_q ? h - kvh * p.gp : 0;
  const bool real = !is_q || in_group < p.g;
  const int64_t src_off = is_q ? (int64_t)(kvh * p.g + in_group) * p.d : (int64_t)kvh * p.d;
  const T* src0 = static_cast<const T*>(is_q ? p.q : p.k) + src_off;
  const int half = p.rot >> 1;
  for (int64_t t = blockIdx.y; t < p.rows; t += gridDim.y) {
    float u[PPL], v[PPL];
    const T* src = src0 + t * p.in_stride;
#pragma unroll
    for (int i = 0; i < PPL; ++i) {
      const int e = (lane + i * 32) * 2;
      u[i] = real && e < p.d ? Elem<T>::load(src + e) : 0.f;
      v[i] = real && e + 1 < p.d ? Elem<T>::load(src + e + 1) : 0.f;
    }
    int64_t slot = -1;
    if (!is_q) {
      slot = p.slots[t];
      if (slot >= p.num_slots) {
        if (lane == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
        slot = -1;
      }
      if (slot < 0) continue;
      // the value is the projection itself
      T* dst = static_cast<T*>(p.v_cache) + (slot * p.hkv + kvh) * p.dp;
#pragma unroll
      for (int i = 0; i < PPL; ++i) {
        const int e = (lane + i * 32) * 2;
        if (e < p.dp) {
          Elem<T>::store(dst + e, u[i]);
          Elem<T>::store(dst + e + 1, v[i]);
        }
      }
    }
    const int64_t pos = p.positions[t];
    const bool pos_ok = pos >= 0 && pos < p.max_position;
    if (!pos_ok && lane == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_POSITION);
    const float* cs = p.cos_sin + (pos_ok ? pos : 0) * p.rot;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PPL; ++i) {
      const int e = lane + i * 32;
      if (e < half) {
        const float c = __ldg(cs + e), s = __ldg(cs + half + e);
        const float a = u[i] * c - v[i] * s, b = v[i] * c + u[i] * s;
        u[i] = a;
        v[i] = b;
      }
      ss += u[i] * u[i] + v[i] * v[i];
    }
    ss = warp_sum(ss);
    const float rs = rsqrtf(ss / (float)p.d + p.eps);
    T* dst = is_q ? static_cast<T*>(p.q_out) + (t * qheads + h) * p.dp
                  : static_cast<T*>(p.k_cache) + (slot * p.hkv + kvh) * p.dp;
#pragma unroll
    for (int i = 0; i < PPL; ++i) {
      const int e = (lane + i * 32) * 2;
      if (e < p.dp) {
        Elem<T>::store(dst + e, u[i] * rs);
        Elem<T>::store(dst + e + 1, v[i] * rs);
      }
    }
  }
}

// bf16, d and dp multiples of 8: LPH = dp / 8 lanes per head, 8 channels (4 pairs) a
// lane, two tokens in flight.
template <int LPH>
__global__ void __launch_bounds__(256) rope_rms_store_vec_kernel(const RopeRmsParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int TOK = 2;
  const int j = threadIdx.x % LPH;
  const int qheads = p.hkv * p.gp;
  const int heads = qheads + p.hkv;
  const int h = blockIdx.x * (256 / LPH) + threadIdx.x / LPH;
  const bool is_q = h < qheads;
  const int kvh = is_q ? h / p.gp : h - qheads;
  const int in_group = is_q ? h - kvh * p.gp : 0;
  const bool live = h < heads;
  const bool real = live && (!is_q || in_group < p.g) && j * 8 < p.d;
  const uint16_t* src = static_cast<const uint16_t*>(is_q ? p.q : p.k) +
                        (is_q ? (int64_t)(kvh * p.g + in_group) : (int64_t)kvh) * p.d + j * 8;
  const int half = p.rot >> 1;
  const bool vec_cs = (half & 3) == 0;
  const float inv_d = 1.0f / (float)p.d;
  for (int64_t t0 = (int64_t)blockIdx.y * TOK; t0 < p.rows; t0 += (int64_t)gridDim.y * TOK) {
    uint4 raw[TOK];
    int64_t slot[TOK], pos[TOK];
    float4 cs[TOK], sn[TOK];
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      raw[i] = make_uint4(0u, 0u, 0u, 0u);
      slot[i] = -1;
      pos[i] = 0;
      if (t0 + i < p.rows) {
        if (real) raw[i] = *reinterpret_cast<const uint4*>(src + (t0 + i) * p.in_stride);
        pos[i] = p.positions[t0 + i];
        if (!is_q) slot[i] = p.slots[t0 + i];
      }
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      if (pos[i] < 0 || pos[i] >= p.max_position) {
        if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_POSITION);
        pos[i] = 0;
      }
      const float* c = p.cos_sin + pos[i] * p.rot;
      cs[i] = make_float4(1.f, 1.f, 1.f, 1.f);
      sn[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      const int e = j * 4;
      if (vec_cs) {
        if (e < half) {
          cs[i] = __ldg(reinterpret_cast<const float4*>(c + e));
          sn[i] = __ldg(reinterpret_cast<const float4*>(c + half + e));
        }
      } else {
        float* cf = reinterpret_cast<float*>(&cs[i]);
        float* sf = reinterpret_cast<float*>(&sn[i]);
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (e + x < half) {
            cf[x] = __ldg(c + e + x);
            sf[x] = __ldg(c + half + e + x);
          }
      }
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      const float u[4] = {bf16lo(raw[i].x), bf16lo(raw[i].y), bf16lo(raw[i].z), bf16lo(raw[i].w)};
      const float v[4] = {bf16hi(raw[i].x), bf16hi(raw[i].y), bf16hi(raw[i].z), bf16hi(raw[i].w)};
      const float c4[4] = {cs[i].x, cs[i].y, cs[i].z, cs[i].w};
      const float s4[4] = {sn[i].x, sn[i].y, sn[i].z, sn[i].w};
      float a[4], b[4], ss = 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        a[x] = u[x] * c4[x] - v[x] * s4[x];
        b[x] = v[x] * c4[x] + u[x] * s4[x];
        ss += a[x] * a[x] + b[x] * b[x];
      }
#pragma unroll
      for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float rs = rsqrtf(ss * inv_d + p.eps);
      if (!live || t0 + i >= p.rows) continue;
      const uint4 r = make_uint4(pack_bf16(a[0] * rs, b[0] * rs), pack_bf16(a[1] * rs, b[1] * rs),
                                 pack_bf16(a[2] * rs, b[2] * rs), pack_bf16(a[3] * rs, b[3] * rs));
      if (is_q) {
        *reinterpret_cast<uint4*>(static_cast<uint16_t*>(p.q_out) +
                                  ((t0 + i) * qheads + h) * p.dp + j * 8) = r;
      } else if (slot[i] >= p.num_slots) {
        if (p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
      } else if (slot[i] >= 0) {
        const int64_t off = (slot[i] * p.hkv + kvh) * p.dp + j * 8;
        *reinterpret_cast<uint4*>(static_cast<uint16_t*>(p.k_cache) + off) = r;
        *reinterpret_cast<uint4*>(static_cast<uint16_t*>(p.v_cache) + off) = raw[i];
      }
    }
  }
}

// act(gate) * up on 8 bf16 at a time
__global__ void __launch_bounds__(256) act_and_mul_bf16x8_kernel(
    const uint16_t* __restrict__ x, int64_t x_stride, uint16_t* __restrict__ out,
    int64_t out_stride, int64_t rows, int packs, int half, int kind) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int TOK = 4;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= packs) return;
  for (int64_t t0 = (int64_t)blockIdx.y * TOK; t0 < rows; t0 += (int64_t)gridDim.y * TOK) {
    uint4 g[TOK], u[TOK];
#pragma unroll
    for (int i = 0; i < TOK; ++i)
      if (t0 + i < rows) {
        const uint16_t* row = x + (t0 + i) * x_stride + c * 8;
        g[i] = *reinterpret_cast<const uint4*>(row);
        u[i] = *reinterpret_cast<const uint4*>(row + half);
      }
#pragma unroll
    for (int i = 0; i < TOK; ++i)
      if (t0 + i < rows)
        *reinterpret_cast<uint4*>(out + (t0 + i) * out_stride + c * 8) =
            make_uint4(act_mul2(g[i].x, u[i].x, kind), act_mul2(g[i].y, u[i].y, kind),
                       act_mul2(g[i].z, u[i].z, kind), act_mul2(g[i].w, u[i].w, kind));
  }
}

__device__ __forceinline__ float act_f32(float g, int kind) {
  return kind == FK_ACT_SILU ? g * sigmoid_f32(g) : gelu_tanh_f32(g);
}

template <typename T>
__global__ void __launch_bounds__(256) act_and_mul_kernel(
    const T* __restrict__ x, int64_t x_stride, T* __restrict__ out, int64_t out_stride,
    int64_t rows, int groups, int half, int kind) {
  pdl_launch_dependents();
  pdl_wait();
  const int g = blockIdx.x * blockDim.x + threadIdx.x;
  if (g >= groups) return;
  for (int64_t t = blockIdx.y; t < rows; t += gridDim.y) {
    const float4 a = Elem<T>::load4(x + t * x_stride + g * 4);
    const float4 b = Elem<T>::load4(x + t * x_stride + half + g * 4);
    Elem<T>::store4(out + t * out_stride + g * 4,
                    make_float4(act_f32(a.x, kind) * b.x, act_f32(a.y, kind) * b.y,
                                act_f32(a.z, kind) * b.z, act_f32(a.w, kind) * b.w));
  }
}

// threads and float4 groups per thread for a row of `groups` float4
static bool row_shape(int groups, int* threads, int* vpt) {
  int v = (groups + 511) / 512;
  v = v <= 1 ? 1 : v <= 2 ? 2 : 4;
  int th = ((groups + v - 1) / v + 31) / 32 * 32;   // no more threads than the row needs
  if (th > 512) th = 512;
  *threads = th;
  *vpt = v;
  return groups <= th * MX_MAX_VPT;
}

template <typename T, bool SHIFT>
static cudaError_t launch_norm_shift(const NormShiftParams& p, int grid, int threads, int vpt,
                                     cudaStream_t s) {
  const dim3 g(grid), b(threads);
  switch (vpt) {
    case 1: return launch_kernel(norm_shift_kernel<T, 1, SHIFT>, g, b, 0, s, p);
    case 2: return launch_kernel(norm_shift_kernel<T, 2, SHIFT>, g, b, 0, s, p);
    default: return launch_kernel(norm_shift_kernel<T, 4, SHIFT>, g, b, 0, s, p);
  }
}
template <typename T>
static cudaError_t launch_combine(const CombineParams& p, int threads, int vpt, cudaStream_t s) {
  const dim3 grid((unsigned)p.rows);
  switch (vpt) {
    case 1: return launch_kernel(branch_combine_kernel<T, 1>, grid, dim3(threads), 0, s, p);
    case 2: return launch_kernel(branch_combine_kernel<T, 2>, grid, dim3(threads), 0, s, p);
    default: return launch_kernel(branch_combine_kernel<T, 4>, grid, dim3(threads), 0, s, p);
  }
}
template <typename T>
static cudaError_t launch_rope_rms(const RopeRmsParams& p, dim3 grid, cudaStream_t s) {
  const int pairs = (p.dp + 1) / 2;
  if (pairs <= 32) return launch_kernel(rope_rms_store_kernel<T, 1>, grid, dim3(256), 0, s, p);
  if (pairs <= 64) return launch_kernel(rope_rms_store_kernel<T, 2>, grid, dim3(256), 0, s, p);
  return launch_kernel(rope_rms_store_kernel<T, 8>, grid, dim3(256), 0, s, p);
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_embed_f32(const void* table, int is_f32, int64_t vocab, const int64_t* ids, float* x,
                 int64_t rows, int stride, int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && vocab > 0 && stride > 0, FK_ERR_INVALID_ARG, "fk_embed_f32: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(table && ids && x, FK_ERR_INVALID_ARG, "fk_embed_f32: null pointer");
  FK_REQUIRE(stride % 8 == 0 && aligned16(table) && aligned16(x), FK_ERR_ALIGNMENT,
             "fk_embed_f32: rows must be 16-byte aligned");
  const int grid = (int)(rows < 4096 ? rows : 4096);
  const int groups = stride / 4;
  const int threads = groups < 256 ? ((groups + 31) / 32) * 32 : 256;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  cudaError_t e = is_f32 ? launch_kernel(embed_f32_kernel<float>, dim3(grid), dim3(threads), 0, s,
                                         (const float*)table, ids, x, rows, groups, vocab, status)
                         : launch_kernel(embed_f32_kernel<uint16_t>, dim3(grid), dim3(threads), 0,
                                         s, (const uint16_t*)table, ids, x, rows, groups, vocab,
                                         status);
  FK_CUDA_OK(e);
  count_launch();
  return FK_OK;
}

int fk_norm_shift(const float* x_in, float* x_out, const void* y, int64_t y_stride,
                  const float* y_gain, const float* gain, const float* shift, void* out,
                  int is_f32, float* state, int num_slots, const int32_t* slots,
                  const int64_t* positions, const int32_t* cu_portions, int num_portions,
                  int64_t rows, int stride, int width, float eps, int32_t* status,
                  fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && width > 0 && stride >= width, FK_ERR_INVALID_ARG,
             "fk_norm_shift: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(x_in && gain && out && (!y || y_gain), FK_ERR_INVALID_ARG,
             "fk_norm_shift: null pointer");
  FK_REQUIRE(!shift || (state && slots && positions && cu_portions && num_portions > 0 &&
                        num_slots > 0 && x_in != x_out),
             FK_ERR_INVALID_ARG,
             "fk_norm_shift: a token shift needs state, slots, positions, portions and a "
             "residual output apart from its input");
  FK_REQUIRE(!y || x_out, FK_ERR_INVALID_ARG, "fk_norm_shift: y needs x_out");
  FK_REQUIRE(stride % 8 == 0 && y_stride % 8 == 0 && aligned16(x_in) && aligned16(x_out) &&
                 aligned16(y) && aligned16(out) && aligned16(shift) && aligned16(state),
             FK_ERR_ALIGNMENT, "fk_norm_shift: rows must be 16-byte aligned");
  int threads, vpt;
  FK_REQUIRE(row_shape(stride / 4, &threads, &vpt), FK_ERR_UNSUPPORTED,
             "fk_norm_shift: width %d too large", width);
  NormShiftParams p{};
  p.x_in = x_in; p.x_out = x_out; p.y = y; p.y_gain = y_gain; p.gain = gain; p.shift = shift;
  p.out = out; p.state = state; p.slots = slots; p.positions = positions; p.cu = cu_portions;
  p.num_portions = num_portions; p.rows = rows; p.y_stride = y_stride; p.stride = stride;
  p.width = width; p.num_slots = num_slots; p.eps = eps; p.status = status;
  // enough rows per CTA to make the recomputed row ahead cheap, enough CTAs to fill
  // the machine
  int rpc = 1;
  if (shift)
    while (rpc < 8 && rows / (rpc * 2) >= 4 * sm_count()) rpc *= 2;
  p.rows_per_cta = rpc;
  const int64_t grid = (rows + rpc - 1) / rpc;
  FK_REQUIRE(grid <= 0x7fffffff, FK_ERR_UNSUPPORTED, "fk_norm_shift: too many rows");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int g = (int)grid;
  FK_CUDA_OK(shift ? (is_f32 ? launch_norm_shift<float, true>(p, g, threads, vpt, s)
                             : launch_norm_shift<uint16_t, true>(p, g, threads, vpt, s))
                   : (is_f32 ? launch_norm_shift<float, false>(p, g, threads, vpt, s)
                             : launch_norm_shift<uint16_t, false>(p, g, threads, vpt, s)));
  count_launch();
  return FK_OK;
}

int fk_branch_combine(const void* a, const void* b, int64_t ab_stride, const float* weight_a,
                      const float* weight_b, const float* gain_out, const float* gain, float* x,
                      void* out, int is_f32, int64_t rows, int stride, int width, float eps,
                      fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && width > 0 && stride >= width, FK_ERR_INVALID_ARG,
             "fk_branch_combine: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(a && b && weight_a && weight_b && gain_out && x && (!out || gain),
             FK_ERR_INVALID_ARG, "fk_branch_combine: null pointer");
  FK_REQUIRE(stride % 8 == 0 && ab_stride % 8 == 0 && aligned16(a) && aligned16(b) &&
                 aligned16(weight_a) && aligned16(weight_b) && aligned16(x) && aligned16(out),
             FK_ERR_ALIGNMENT, "fk_branch_combine: rows must be 16-byte aligned");
  int threads, vpt;
  FK_REQUIRE(row_shape(stride / 4, &threads, &vpt) && rows <= 0x7fffffff, FK_ERR_UNSUPPORTED,
             "fk_branch_combine: width %d or row count too large", width);
  CombineParams p{};
  p.a = a; p.b = b; p.wa = weight_a; p.wb = weight_b; p.gain_out = gain_out; p.gain = gain;
  p.x = x; p.out = out; p.rows = rows; p.ab_stride = ab_stride; p.stride = stride;
  p.width = width; p.eps = eps;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32 ? launch_combine<float>(p, threads, vpt, s)
                    : launch_combine<uint16_t>(p, threads, vpt, s));
  count_launch();
  return FK_OK;
}

int fk_rope_rms_store(const void* q, const void* k, int64_t in_stride, int is_f32, void* q_out,
                      void* k_cache, void* v_cache, const int32_t* slots, int64_t num_slots,
                      const int64_t* positions, const float* cos_sin, int64_t max_position,
                      int rot_dims, int num_q_heads, int num_kv_heads, int head_dim,
                      int padded_group, int padded_dim, float eps, int64_t rows,
                      int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && num_kv_heads > 0 && num_q_heads > 0 && head_dim > 0,
             FK_ERR_INVALID_ARG, "fk_rope_rms_store: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(num_q_heads % num_kv_heads == 0, FK_ERR_INVALID_ARG,
             "fk_rope_rms_store: num_q_heads must be a multiple of num_kv_heads");
  FK_REQUIRE(q && k && q_out && k_cache && v_cache && slots && positions && cos_sin,
             FK_ERR_INVALID_ARG, "fk_rope_rms_store: null pointer");
  FK_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= head_dim &&
                 padded_dim >= head_dim && padded_dim % 2 == 0 &&
                 padded_group >= num_q_heads / num_kv_heads,
             FK_ERR_INVALID_ARG, "fk_rope_rms_store: bad rotation or padding sizes");
  FK_REQUIRE(padded_dim <= 512, FK_ERR_UNSUPPORTED,
             "fk_rope_rms_store: head size %d too large", head_dim);
  RopeRmsParams p{};
  p.q = q; p.k = k; p.in_stride = in_stride; p.q_out = q_out; p.k_cache = k_cache;
  p.v_cache = v_cache; p.slots = slots; p.num_slots = num_slots; p.positions = positions;
  p.cos_sin = cos_sin; p.max_position = max_position; p.rot = rot_dims; p.hkv = num_kv_heads;
  p.g = num_q_heads / num_kv_heads; p.gp = padded_group; p.d = head_dim; p.dp = padded_dim;
  p.eps = eps; p.rows = rows; p.status = status;
  const int heads = num_kv_heads * (padded_group + 1);
  const int64_t ny = rows < 8192 ? rows : 8192;
  const dim3 grid((unsigned)((heads + 7) / 8), (unsigned)ny);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = !is_f32 && head_dim % 8 == 0 && (padded_dim == 64 || padded_dim == 128) &&
                   in_stride % 8 == 0 && aligned16(q) && aligned16(k) && aligned16(q_out) &&
                   aligned16(k_cache) && aligned16(v_cache) && aligned16(cos_sin);
  if (vec) {
    const int per = 256 / (padded_dim / 8);
    const int gx = (heads + per - 1) / per;
    const int64_t pairs = (rows + 1) / 2;
    int64_t gy = (int64_t)sm_count() * 16 / gx;
    gy = gy < 1 ? 1 : gy < pairs ? gy : pairs;
    const dim3 vgrid((unsigned)gx, (unsigned)gy);
    FK_CUDA_OK(padded_dim == 64
                   ? launch_kernel(rope_rms_store_vec_kernel<8>, vgrid, dim3(256), 0, s, p)
                   : launch_kernel(rope_rms_store_vec_kernel<16>, vgrid, dim3(256), 0, s, p));
    count_launch();
    return FK_OK;
  }
  FK_CUDA_OK(is_f32 ? launch_rope_rms<float>(p, grid, s) : launch_rope_rms<uint16_t>(p, grid, s));
  count_launch();
  return FK_OK;
}

int fk_act_and_mul(const void* x, int64_t x_stride, void* out, int64_t out_stride, int is_f32,
                   int64_t rows, int64_t d, int act, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && d > 0, FK_ERR_INVALID_ARG, "fk_act_and_mul: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(x && out, FK_ERR_INVALID_ARG, "fk_act_and_mul: null pointer");
  FK_REQUIRE(act == FK_ACT_SILU || act == FK_ACT_GELU_TANH, FK_ERR_INVALID_ARG,
             "fk_act_and_mul: unknown activation %d", act);
  FK_REQUIRE(d % 8 == 0 && x_stride % 8 == 0 && out_stride % 8 == 0 && aligned16(x) &&
                 aligned16(out),
             FK_ERR_ALIGNMENT, "fk_act_and_mul: rows must be 16-byte aligned");
  FK_REQUIRE(d < (1ll << 30) && x_stride >= 2 * d && out_stride >= d, FK_ERR_INVALID_ARG,
             "fk_act_and_mul: bad stride");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (is_f32) {
    const int groups = (int)(d / 4);
    const dim3 grid((unsigned)((groups + 255) / 256), (unsigned)(rows < 16384 ? rows : 16384));
    e = launch_kernel(act_and_mul_kernel<float>, grid, dim3(256), 0, s, (const float*)x, x_stride,
                      (float*)out, out_stride, rows, groups, (int)d, act);
  } else {
    const int packs = (int)(d / 8);
    const int64_t quads = (rows + 3) / 4;
    const dim3 grid((unsigned)((packs + 255) / 256), (unsigned)(quads < 16384 ? quads : 16384));
    e = launch_kernel(act_and_mul_bf16x8_kernel, grid, dim3(256), 0, s, (const uint16_t*)x,
                      x_stride, (uint16_t*)out, out_stride, rows, packs, (int)d, act);
  }
  FK_CUDA_OK(e);
  count_launch();
  return FK_OK;
}

}  // extern "C"
