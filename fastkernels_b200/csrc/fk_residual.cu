// Row kernels of decoders with an fp32 residual stream whose sublayers run side by side:
//
//   fk_embed_pair_f32     embedding row + a row chosen by (previous token, token)
//   fk_add_layernorm      residual += sublayer outputs (dense ones and the weighted rows
//                         of a mixture of experts), then up to two layer norms of it
//   fk_head_norm_gate     per-head RMS norm, weight, sigmoid gate (recurrent mixers)
//   fk_softcap            cap * tanh(z / cap) in place
//
// bf16 and fp32 activations; rows padded with a zero tail, so every access is a full
// vector.  All of them are bound by HBM traffic.
#include "fk_types.cuh"

namespace fk {

struct EmbedPairParams {
  const void* table; const void* pairs;     // [vocab, stride], [buckets + 1, stride] or null
  int64_t vocab, buckets, mul_prev, mul_cur;
  const int64_t* ids;
  int64_t* last;                            // [slots]: last token of a sequence
  const int32_t* slots; const int64_t* positions;
  const int32_t* cu; int num_portions, num_slots;
  float* x; void* copy; int64_t copy_stride;
  int64_t rows; int groups;
  int32_t* status;
};

// Row of the pair table: (prev * mul_prev + token * mul_cur) mod buckets, the last row for
// a sequence's first token.  The CTA that owns a portion's first row reads the sequence's
// last token AND replaces it by the portion's last one: nobody else touches it.
template <typename T>
__global__ void __launch_bounds__(256) embed_pair_kernel(const EmbedPairParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int64_t row_of;
  for (int64_t t = blockIdx.x; t < p.rows; t += gridDim.x) {
    const int64_t id = p.ids[t];
    const bool ok = id >= 0 && id < p.vocab;
    if (threadIdx.x == 0) {
      if (!ok && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
      int64_t prev = -1;
      if (p.pairs) {
        const int slot = p.slots[t];
        const bool first = t == 0 || slot < 0 || p.slots[t - 1] != slot;
        if (!first) {
          prev = p.ids[t - 1];
        } else if (slot >= p.num_slots) {
          if (p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
        } else if (slot >= 0) {
          if (p.positions[t] > 0) prev = p.last[slot];
          int lo = 0, hi = p.num_portions;
          while (hi - lo > 1) {
            const int mid = (lo + hi) >> 1;
            if (p.cu[mid] <= t) lo = mid; else hi = mid;
          }
          const int64_t end = min((int64_t)p.cu[lo + 1], p.rows);
          p.last[slot] = p.ids[max(t, end - 1)];
        }
      }
      int64_t r = p.buckets;
      if (prev >= 0) {
        r = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
        if (r < 0) r += p.buckets;
      }
      row_of = r;
    }
    __syncthreads();
    const int64_t r = row_of;
    __syncthreads();
    for (int g = threadIdx.x; g < p.groups; g += blockDim.x) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (ok) {
        v = Elem<T>::load4(static_cast<const T*>(p.table) + (id * p.groups + g) * 4);
        if (p.pairs)
          v = v + Elem<T>::load4(static_cast<const T*>(p.pairs) + (r * p.groups + g) * 4);
      }
      *reinterpret_cast<float4*>(p.x + (t * p.groups + g) * 4) = v;
      if (p.copy) Elem<T>::store4(static_cast<T*>(p.copy) + t * p.copy_stride + g * 4, v);
    }
  }
}

struct AddLayerNormParams {
  const float* x_in; float* x_out;          // [T, stride]; x_out null: not stored
  const void* a; const void* b;             // [T, a_stride] / [T, b_stride] or null
  const void* e; const int32_t* place; const float* share; int top;   // expert rows
  const float* w1; const float* b1; void* out1;   // w1 null: out1 = the sum itself
  const float* w2; const float* b2; void* out2;   // null: one norm only
  int64_t rows, a_stride, b_stride, e_stride, e_rows, out1_stride, out2_stride;
  int stride, width;
  float eps;
  int32_t* status;
};

template <typename T, int VPT>
__global__ void __launch_bounds__(512) add_layernorm_kernel(const AddLayerNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[64];
  int flip = 0;
  const int groups = p.stride >> 2;
  const float inv_w = 1.0f / (float)p.width;
  for (int64_t t = blockIdx.x; t < p.rows; t += gridDim.x) {
    float4 x[VPT];
    float s[1] = {0.f};
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int g = threadIdx.x + i * blockDim.x;
      x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (g < groups) {
        x[i] = *reinterpret_cast<const float4*>(p.x_in + t * p.stride + g * 4);
        if (p.a) x[i] = x[i] + Elem<T>::load4(static_cast<const T*>(p.a) + t * p.a_stride + g * 4);
        if (p.b) x[i] = x[i] + Elem<T>::load4(static_cast<const T*>(p.b) + t * p.b_stride + g * 4);
      }
    }
    if (p.e) {
      for (int j = 0; j < p.top; ++j) {
        const int64_t r = p.place[t * p.top + j];
        if (r < 0 || r >= p.e_rows) {
          if (threadIdx.x == 0 && p.status) atomicOr(p.status, FK_DEV_BAD_SLOT);
          continue;
        }
        const float wj = p.share[t * p.top + j];
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int g = threadIdx.x + i * blockDim.x;
          if (g < groups)
            x[i] = x[i] + Elem<T>::load4(static_cast<const T*>(p.e) + r * p.e_stride + g * 4) * wj;
        }
      }
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int g = threadIdx.x + i * blockDim.x;
      if (g < groups && p.x_out)
        *reinterpret_cast<float4*>(p.x_out + t * p.stride + g * 4) = x[i];
      s[0] += (x[i].x + x[i].y) + (x[i].z + x[i].w);   // the tail is zero
    }
    if (!p.w1) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int g = threadIdx.x + i * blockDim.x;
        if (g < groups && p.out1)
          Elem<T>::store4(static_cast<T*>(p.out1) + t * p.out1_stride + g * 4, x[i]);
      }
      continue;
    }
    block_sums<1>(s, red, flip);
    const float mu = s[0] * inv_w;
    float v[1] = {0.f};
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 4;
      x[i] = make_float4(c < p.width ? x[i].x - mu : 0.f, c + 1 < p.width ? x[i].y - mu : 0.f,
                         c + 2 < p.width ? x[i].z - mu : 0.f, c + 3 < p.width ? x[i].w - mu : 0.f);
      v[0] += sumsq(x[i]);
    }
    block_sums<1>(v, red, flip);
    const float rs = 1.0f / sqrtf(v[0] * inv_w + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int g = threadIdx.x + i * blockDim.x;
      if (g >= groups) continue;
      const float4 n = x[i] * rs;
      Elem<T>::store4(static_cast<T*>(p.out1) + t * p.out1_stride + g * 4,
                      n * __ldg(reinterpret_cast<const float4*>(p.w1 + g * 4)) +
                          __ldg(reinterpret_cast<const float4*>(p.b1 + g * 4)));
      if (p.out2)
        Elem<T>::store4(static_cast<T*>(p.out2) + t * p.out2_stride + g * 4,
                        n * __ldg(reinterpret_cast<const float4*>(p.w2 + g * 4)) +
                            __ldg(reinterpret_cast<const float4*>(p.b2 + g * 4)));
    }
  }
}

template <typename T>
static cudaError_t launch_add_layernorm(const AddLayerNormParams& p, cudaStream_t s) {
  const int groups = p.stride / 4;
  // many rows: several vectors a thread, so that a CTA has few warps to bring together
  int vpt = (groups + 511) / 512;
  if (p.rows >= 2 * sm_count()) vpt = groups >= 512 ? 4 : groups >= 128 ? 2 : 1;
  vpt = vpt <= 1 ? 1 : vpt <= 2 ? 2 : vpt <= 4 ? 4 : 8;
  int threads = ((groups + vpt - 1) / vpt + 31) / 32 * 32;
  while (threads > 512) { vpt *= 2; threads = ((groups + vpt - 1) / vpt + 31) / 32 * 32; }
  const int64_t cap = (int64_t)sm_count() * 64;
  const dim3 grid((unsigned)(p.rows < cap ? p.rows : cap)), block((unsigned)threads);
  switch (vpt) {
    case 1: return launch_kernel(add_layernorm_kernel<T, 1>, grid, block, 0, s, p);
    case 2: return launch_kernel(add_layernorm_kernel<T, 2>, grid, block, 0, s, p);
    case 4: return launch_kernel(add_layernorm_kernel<T, 4>, grid, block, 0, s, p);
    default: return launch_kernel(add_layernorm_kernel<T, 8>, grid, block, 0, s, p);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) softcap_kernel(T* __restrict__ x, int64_t stride,
                                                      int64_t rows, int64_t cols, float cap,
                                                      bool vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t c = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= cols) return;
  const float inv = 1.0f / cap;
  for (int64_t t = blockIdx.y; t < rows; t += gridDim.y) {
    T* q = x + t * stride + c;
    if (vec && c + 4 <= cols) {
      const float4 v = Elem<T>::load4(q);
      Elem<T>::store4(q, make_float4(cap * tanhf(v.x * inv), cap * tanhf(v.y * inv),
                                     cap * tanhf(v.z * inv), cap * tanhf(v.w * inv)));
    } else {
      for (int i = 0; i < 4 && c + i < cols; ++i)
        Elem<T>::store(q + i, cap * tanhf(Elem<T>::load(q + i) * inv));
    }
  }
}

constexpr int HN_MAX_DIM = 1024;

struct HeadNormParams {
  const float* o;                     // [rows][heads * d]
  const void* g; int64_t g_stride;    // gate projection
  const float* weight;                // [heads * d]
  void* out; int64_t out_stride;      // [rows, out_stride], tail beyond heads * d zeroed
  int64_t rows; int heads, d;
  float eps;
};

// d a multiple of 4: LPH lanes per (token, head), NV groups of four channels a lane.
template <typename T, int LPH, int NV>
__global__ void __launch_bounds__(256) head_norm_gate_vec_kernel(const HeadNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int PER = 256 / LPH;                 // (token, head) pairs per CTA and pass
  const int j = threadIdx.x % LPH;
  const int h = blockIdx.x * PER + threadIdx.x / LPH;
  const int64_t hd = (int64_t)p.heads * p.d;
  const int64_t c0 = (int64_t)h * p.d + j * 4;
  bool on[NV];
  float4 wt[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    on[i] = h < p.heads && (j + i * LPH) * 4 < p.d;
    wt[i] = on[i] ? __ldg(reinterpret_cast<const float4*>(p.weight + c0 + i * LPH * 4))
                  : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int64_t t = blockIdx.y; t < p.rows; t += gridDim.y) {
    float4 x[NV], g[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      x[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (on[i]) {
        x[i] = *reinterpret_cast<const float4*>(p.o + t * hd + c0 + i * LPH * 4);
        g[i] = Elem<T>::load4(static_cast<const T*>(p.g) + t * p.g_stride + c0 + i * LPH * 4);
      }
      ss += sumsq(x[i]);
    }
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rs = rsqrtf(ss / (float)p.d + p.eps);
    T* out = static_cast<T*>(p.out) + t * p.out_stride;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (on[i])
        Elem<T>::store4(out + c0 + i * LPH * 4,
                        (x[i] * rs) * wt[i] *
                            make_float4(sigmoid_f32(g[i].x), sigmoid_f32(g[i].y),
                                        sigmoid_f32(g[i].z), sigmoid_f32(g[i].w)));
    if (blockIdx.x == 0 && hd + threadIdx.x < p.out_stride && threadIdx.x < 64)
      Elem<T>::store(out + hd + threadIdx.x, 0.f);
  }
}

// One warp per (token, head), any d.
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const HeadNormParams p) {
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
    float x[HN_MAX_DIM / 32];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < HN_MAX_DIM / 32; ++i) {
      const int c = lane + i * 32;
      x[i] = c < p.d ? o[c] : 0.f;
      ss += x[i] * x[i];
    }
    ss = warp_sum(ss);
    const float rs = rsqrtf(ss / (float)p.d + p.eps);
#pragma unroll
    for (int i = 0; i < HN_MAX_DIM / 32; ++i) {
      const int c = lane + i * 32;
      if (c < p.d)
        Elem<T>::store(out + (int64_t)h * p.d + c,
                       x[i] * rs * p.weight[(int64_t)h * p.d + c] *
                           sigmoid_f32(Elem<T>::load(g + c)));
    }
  }
}

template <typename T, int LPH, int NV = 1>
static cudaError_t launch_head_norm_vec(const HeadNormParams& p, cudaStream_t s) {
  constexpr int PER = 256 / LPH;
  const int gx = (p.heads + PER - 1) / PER;
  int64_t gy = (int64_t)sm_count() * 8 / gx;       // CTAs resident at once, tokens strided
  gy = gy < 1 ? 1 : gy < p.rows ? gy : p.rows;
  return launch_kernel(head_norm_gate_vec_kernel<T, LPH, NV>, dim3((unsigned)gx, (unsigned)gy),
                       dim3(256), 0, s, p);
}
template <typename T>
static cudaError_t launch_head_norm(const HeadNormParams& p, bool vec, cudaStream_t s) {
  if (vec && p.d <= 32) return launch_head_norm_vec<T, 8>(p, s);
  if (vec && p.d <= 64) return launch_head_norm_vec<T, 16>(p, s);
  if (vec && p.d <= 128) return launch_head_norm_vec<T, 32>(p, s);
  if (vec && p.d <= 256) return launch_head_norm_vec<T, 32, 2>(p, s);
  if (vec && p.d <= 512) return launch_head_norm_vec<T, 32, 4>(p, s);
  const dim3 grid((unsigned)(p.heads / 8 + 1), (unsigned)(p.rows < 8192 ? p.rows : 8192));
  return launch_kernel(head_norm_gate_kernel<T>, grid, dim3(256), 0, s, p);
}

}  // namespace fk

using namespace fk;

extern "C" {

int fk_embed_pair_f32(const void* table, const void* pairs, int is_f32, int64_t vocab,
                      int64_t buckets, int64_t mul_prev, int64_t mul_cur, const int64_t* ids,
                      int64_t* last_ids, int num_slots, const int32_t* slots,
                      const int64_t* positions, const int32_t* cu_portions, int num_portions,
                      float* x, void* copy, int64_t copy_stride, int64_t rows, int stride,
                      int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && vocab > 0 && stride > 0, FK_ERR_INVALID_ARG,
             "fk_embed_pair_f32: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(table && ids && x, FK_ERR_INVALID_ARG, "fk_embed_pair_f32: null pointer");
  FK_REQUIRE(!pairs || (buckets > 0 && last_ids && slots && positions && cu_portions &&
                        num_portions > 0 && num_slots > 0),
             FK_ERR_INVALID_ARG,
             "fk_embed_pair_f32: a pair table needs buckets, last tokens, slots, positions and "
             "portions");
  FK_REQUIRE(stride % 8 == 0 && (!copy || (copy_stride >= stride && copy_stride % 8 == 0)) &&
                 aligned16(table) && aligned16(pairs) && aligned16(x) && aligned16(copy),
             FK_ERR_ALIGNMENT, "fk_embed_pair_f32: rows must be 16-byte aligned");
  EmbedPairParams p{};
  p.table = table; p.pairs = pairs; p.vocab = vocab; p.buckets = buckets; p.mul_prev = mul_prev;
  p.mul_cur = mul_cur; p.ids = ids; p.last = last_ids; p.slots = slots; p.positions = positions;
  p.cu = cu_portions; p.num_portions = num_portions; p.num_slots = num_slots; p.x = x;
  p.copy = copy; p.copy_stride = copy_stride; p.rows = rows; p.groups = stride / 4;
  p.status = status;
  const int grid = (int)(rows < 8192 ? rows : 8192);
  const int threads = p.groups < 256 ? ((p.groups + 31) / 32) * 32 : 256;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32 ? launch_kernel(embed_pair_kernel<float>, dim3(grid), dim3(threads), 0, s, p)
                    : launch_kernel(embed_pair_kernel<uint16_t>, dim3(grid), dim3(threads), 0, s,
                                    p));
  count_launch();
  return FK_OK;
}

int fk_add_layernorm(const float* x_in, float* x_out, const void* a, int64_t a_stride,
                     const void* b, int64_t b_stride, const void* experts, int64_t expert_stride,
                     int64_t expert_rows, const int32_t* place, const float* share, int top,
                     const float* weight1, const float* bias1, void* out1, int64_t out1_stride,
                     const float* weight2, const float* bias2, void* out2, int64_t out2_stride,
                     int is_f32, int64_t rows, int stride, int width, float eps,
                     int32_t* status, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && width > 0 && stride >= width, FK_ERR_INVALID_ARG,
             "fk_add_layernorm: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(x_in && (x_out || out1) && (!weight1 || (bias1 && out1)) &&
                 (!out2 || (weight1 && weight2 && bias2)) &&
                 (!experts || (place && share && top > 0)),
             FK_ERR_INVALID_ARG, "fk_add_layernorm: null pointer");
  FK_REQUIRE(stride % 8 == 0 && (!a || a_stride % 4 == 0) && (!b || b_stride % 4 == 0) &&
                 (!experts || expert_stride % 4 == 0) && (!out1 || out1_stride % 4 == 0) &&
                 (!out2 || out2_stride % 4 == 0) && aligned16(x_in) && aligned16(x_out) &&
                 aligned16(a) && aligned16(b) && aligned16(experts) && aligned16(out1) &&
                 aligned16(out2) && aligned16(weight1) && aligned16(bias1) &&
                 aligned16(weight2) && aligned16(bias2),
             FK_ERR_ALIGNMENT, "fk_add_layernorm: rows must be 16-byte aligned");
  FK_REQUIRE((!a || a_stride >= stride) && (!b || b_stride >= stride) &&
                 (!experts || expert_stride >= stride) && (!out1 || out1_stride >= stride) &&
                 (!out2 || out2_stride >= stride),
             FK_ERR_INVALID_ARG, "fk_add_layernorm: row stride smaller than the row");
  FK_REQUIRE(stride <= 16384, FK_ERR_UNSUPPORTED, "fk_add_layernorm: width %d too large", width);
  AddLayerNormParams p{};
  p.x_in = x_in; p.x_out = x_out; p.a = a; p.b = b; p.e = experts; p.place = place;
  p.share = share; p.top = top; p.w1 = weight1; p.b1 = bias1; p.out1 = out1; p.w2 = weight2;
  p.b2 = bias2; p.out2 = out2; p.rows = rows; p.a_stride = a_stride; p.b_stride = b_stride;
  p.e_stride = expert_stride; p.e_rows = expert_rows; p.out1_stride = out1_stride;
  p.out2_stride = out2_stride; p.stride = stride; p.width = width; p.eps = eps; p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  FK_CUDA_OK(is_f32 ? launch_add_layernorm<float>(p, s) : launch_add_layernorm<uint16_t>(p, s));
  count_launch();
  return FK_OK;
}

int fk_softcap(void* x, int64_t stride, int is_f32, int64_t rows, int64_t cols, float cap,
               fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && cols >= 0 && cap > 0.f, FK_ERR_INVALID_ARG, "fk_softcap: bad sizes");
  if (rows == 0 || cols == 0) return FK_OK;
  FK_REQUIRE(x && stride >= cols, FK_ERR_INVALID_ARG, "fk_softcap: null pointer or bad stride");
  FK_REQUIRE(cols <= (1ll << 31), FK_ERR_UNSUPPORTED, "fk_softcap: row too long");
  const dim3 grid((unsigned)((cols + 1023) / 1024), (unsigned)(rows < 65535 ? rows : 65535));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = stride % 4 == 0 && aligned16(x);
  FK_CUDA_OK(is_f32 ? launch_kernel(softcap_kernel<float>, grid, dim3(256), 0, s, (float*)x,
                                    stride, rows, cols, cap, vec)
                    : launch_kernel(softcap_kernel<uint16_t>, grid, dim3(256), 0, s, (uint16_t*)x,
                                    stride, rows, cols, cap, vec));
  count_launch();
  return FK_OK;
}

int fk_head_norm_gate(const float* o, const void* gate, int64_t gate_stride, const float* weight,
                    void* out, int64_t out_stride, int is_f32, int64_t rows, int heads, int dim,
                    float eps, fk_stream_t stream) {
  FK_REQUIRE(rows >= 0 && heads > 0 && dim > 0, FK_ERR_INVALID_ARG,
             "fk_head_norm_gate: bad sizes");
  if (rows == 0) return FK_OK;
  FK_REQUIRE(o && gate && weight && out, FK_ERR_INVALID_ARG, "fk_head_norm_gate: null pointer");
  FK_REQUIRE(dim <= HN_MAX_DIM, FK_ERR_UNSUPPORTED, "fk_head_norm_gate: head size %d too large",
             dim);
  FK_REQUIRE(out_stride >= (int64_t)heads * dim && gate_stride >= (int64_t)heads * dim,
             FK_ERR_INVALID_ARG, "fk_head_norm_gate: bad stride");
  HeadNormParams p{};
  p.o = o; p.g = gate; p.g_stride = gate_stride; p.weight = weight; p.out = out;
  p.out_stride = out_stride; p.rows = rows; p.heads = heads; p.d = dim; p.eps = eps;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = dim % 4 == 0 && dim <= 512 && gate_stride % 4 == 0 && out_stride % 4 == 0 &&
                   out_stride - (int64_t)heads * dim <= 64 && aligned16(o) && aligned16(gate) &&
                   aligned16(weight) && aligned16(out);
  FK_CUDA_OK(is_f32 ? launch_head_norm<float>(p, vec, s) : launch_head_norm<uint16_t>(p, vec, s));
  count_launch();
  return FK_OK;
}

}  // extern "C"
