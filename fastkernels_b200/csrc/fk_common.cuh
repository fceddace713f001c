// Shared host/device helpers for the fk_b200 kernels (sm_100a only).
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <atomic>
#include <cstdarg>
#include <cstdio>

#include "../../include/fk_b200.h"

namespace fk {

// ---------------------------------------------------------------- host side
void set_error(const char* fmt, ...);
void count_launch(int n = 1);

#define FK_REQUIRE(cond, code, ...)  \
  do {                               \
    if (!(cond)) {                   \
      ::fk::set_error(__VA_ARGS__);  \
      return (code);                 \
    }                                \
  } while (0)

#define FK_CUDA_OK(expr)                                                   \
  do {                                                                     \
    cudaError_t e__ = (expr);                                              \
    if (e__ != cudaSuccess) {                                              \
      ::fk::set_error("%s failed: %s", #expr, cudaGetErrorString(e__));    \
      return FK_ERR_CUDA;                                                  \
    }                                                                      \
  } while (0)

inline bool aligned16(const void* p) {
  return (reinterpret_cast<uintptr_t>(p) & 15u) == 0;
}

// Programmatic dependent launch: when enabled (default), every kernel of the
// library is launched with the programmatic-stream-serialization attribute, lets
// its successor start early (griddepcontrol.launch_dependents at its top) and
// waits for its predecessors (griddepcontrol.wait) before it touches memory they
// may have written.  The successor's launch latency, prologue and -- in the GEMM
// -- its first weight tiles then overlap the tail of the running kernel.
bool pdl_enabled();

template <typename... KArgs, typename... Args>
inline cudaError_t launch_kernel_pdl(bool early, void (*kernel)(KArgs...), dim3 grid, dim3 block,
                                     size_t smem, cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = early && pdl_enabled() ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
template <typename... KArgs, typename... Args>
inline cudaError_t launch_kernel(void (*kernel)(KArgs...), dim3 grid, dim3 block,
                                 size_t smem, cudaStream_t stream, Args... args) {
  return launch_kernel_pdl(true, kernel, grid, block, smem, stream, args...);
}
// For a kernel whose CTAs should find empty SMs: it starts when its predecessors have
// ended.
template <typename... KArgs, typename... Args>
inline cudaError_t launch_kernel_after(void (*kernel)(KArgs...), dim3 grid, dim3 block,
                                       size_t smem, cudaStream_t stream, Args... args) {
  return launch_kernel_pdl(false, kernel, grid, block, smem, stream, args...);
}

#define FK_LAUNCH(kernel, ...) (void)::fk::launch_kernel(kernel, __VA_ARGS__)

// Number of SMs of the current device (cached per device).
int sm_count();

// A function attribute such as the dynamic shared-memory limit belongs to ONE
// device's copy of the kernel, so a process that drives several GPUs has to set
// it on each of them: `set_max_dynamic_smem` does it on the first launch per
// (kernel, device) and remembers which devices are done in a bit mask.
struct PerDeviceOnce {
  std::atomic<uint64_t> done{0};
};
template <typename K>
inline cudaError_t set_max_dynamic_smem(PerDeviceOnce& once, K kernel, int bytes) {
  int dev = -1;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  const bool tracked = dev >= 0 && dev < 64;
  if (tracked && (once.done.load(std::memory_order_acquire) >> dev) & 1ull)
    return cudaSuccess;
  e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e == cudaSuccess && tracked)
    once.done.fetch_or(1ull << dev, std::memory_order_release);
  return e;
}

// cuTensorMapEncodeTiled resolved through the runtime (no libcuda link).
typedef CUresult (*tensormap_encode_fn)(
    CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
    const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
    CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion,
    CUtensorMapFloatOOBfill);
tensormap_encode_fn get_tensormap_encode();

// -------------------------------------------------------------- device side
#ifdef __CUDACC__

__device__ __forceinline__ float bf16_bits_to_float(uint32_t lo16) {
  return __uint_as_float(lo16 << 16);
}
__device__ __forceinline__ float bf16lo(uint32_t packed) {
  return __uint_as_float(packed << 16);
}
__device__ __forceinline__ float bf16hi(uint32_t packed) {
  return __uint_as_float(packed & 0xffff0000u);
}
// Round-to-nearest-even fp32 -> bf16, two values packed (lo = a, hi = b).
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  uint32_t r;
  asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r) : "f"(b), "f"(a));
  return r;
}
__device__ __forceinline__ float round_bf16(float a) {
  return __bfloat162float(__float2bfloat16_rn(a));
}

// ---- SiLU-and-multiply on packed bf16 pairs ----------------------------------
// reference: fastkernels/tasks/baseline/L1/silu_and_mul.cu:715-740, 823-830
//   out = bf16(float(bf16(g / (1 + exp(-g)))) * float(u))
// The quotient is rounded to bf16 right away (8 significant bits), so the
// hardware exponential and reciprocal (relative error ~2^-21) stand in for the
// exact ones: the rounded value differs in well under one element per thousand,
// and then by one bf16 step.  It takes the arithmetic per element from ~20
// instructions to 6, which matters at 50 M elements per call.
__device__ __forceinline__ float silu_f32(float g) {
  return __fdividef(g, 1.0f + __expf(-g));
}
__device__ __forceinline__ uint32_t silu_mul2(uint32_t g, uint32_t u) {
  const float g0 = bf16lo(g), g1 = bf16hi(g);
  const float a0 = round_bf16(silu_f32(g0));
  const float a1 = round_bf16(silu_f32(g1));
  return pack_bf16(a0 * bf16lo(u), a1 * bf16hi(u));
}

// Tanh-form GELU, 0.5 g (1 + tanh(a)) = g sigmoid(2 a) with
// a = sqrt(2 / pi) (g + 0.044715 g^3).
__device__ __forceinline__ float gelu_tanh_arg(float g) {
  return 1.5957691216057308f * (g + 0.044715f * g * g * g);   // 2 a
}
__device__ __forceinline__ float gelu_tanh_f32(float g) {
  return g / (1.0f + expf(-gelu_tanh_arg(g)));
}
// The same on packed bf16 pairs times `u`, rounded once at the end.
__device__ __forceinline__ uint32_t gelu_mul2(uint32_t g, uint32_t u) {
  const float g0 = bf16lo(g), g1 = bf16hi(g);
  const float a0 = __fdividef(g0, 1.0f + __expf(-gelu_tanh_arg(g0)));
  const float a1 = __fdividef(g1, 1.0f + __expf(-gelu_tanh_arg(g1)));
  return pack_bf16(a0 * bf16lo(u), a1 * bf16hi(u));
}
__device__ __forceinline__ uint32_t act_mul2(uint32_t g, uint32_t u, int act) {
  return act == FK_ACT_GELU_TANH ? gelu_mul2(g, u) : silu_mul2(g, u);
}

// No-ops when the kernel was launched without the programmatic attribute.
__device__ __forceinline__ void pdl_launch_dependents() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}
__device__ __forceinline__ void pdl_wait() {
  asm volatile("griddepcontrol.wait;" ::: "memory");
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

// ---- mbarrier -------------------------------------------------------------
__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)),
               "r"(count)
               : "memory");
}
__device__ __forceinline__ void mbar_fence_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void mbar_arrive_expect_tx(uint64_t* bar,
                                                      uint32_t bytes) {
  asm volatile(
      "mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(
          smem_u32(bar)),
      "r"(bytes)
      : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}
// Bounded wait: returns false when the limit ran out (caller records
// FK_DEV_WAIT_TIMEOUT and unwinds; nothing spins forever).
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity,
                                          uint32_t limit = (1u << 24)) {
  for (uint32_t i = 0; i < limit; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
  }
  return false;
}

// ---- TMA ------------------------------------------------------------------
__device__ __forceinline__ void tma_prefetch_desc(const CUtensorMap* m) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(m) : "memory");
}
__device__ __forceinline__ void tma_load_4d(void* dst, const CUtensorMap* m,
                                            uint64_t* bar, int c0, int c1,
                                            int c2, int c3) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cta.global.mbarrier::complete_tx::bytes"
      " [%0], [%1, {%3, %4, %5, %6}], [%2];" ::"r"(smem_u32(dst)),
      "l"(m), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3)
      : "memory");
}
__device__ __forceinline__ void tma_load_5d(void* dst, const CUtensorMap* m,
                                            uint64_t* bar, int c0, int c1,
                                            int c2, int c3, int c4) {
  asm volatile(
      "cp.async.bulk.tensor.5d.shared::cta.global.mbarrier::complete_tx::bytes"
      " [%0], [%1, {%3, %4, %5, %6, %7}], [%2];" ::"r"(smem_u32(dst)),
      "l"(m), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(c4)
      : "memory");
}
__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* m,
                                            uint64_t* bar, int c0, int c1) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cta.global.mbarrier::complete_tx::bytes"
      " [%0], [%1, {%3, %4}], [%2];" ::"r"(smem_u32(dst)),
      "l"(m), "r"(smem_u32(bar)), "r"(c0), "r"(c1)
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* m,
                                            uint64_t* bar, int c0, int c1, int c2) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cta.global.mbarrier::complete_tx::bytes"
      " [%0], [%1, {%3, %4, %5}], [%2];" ::"r"(smem_u32(dst)),
      "l"(m), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
// Untiled bulk copy global -> shared (both 16-byte aligned, size % 16 == 0).
__device__ __forceinline__ void bulk_load(void* dst, const void* src,
                                          uint32_t bytes, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.shared::cta.global.mbarrier::complete_tx::bytes"
      " [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
      "l"(src), "r"(bytes), "r"(smem_u32(bar))
      : "memory");
}
__device__ __forceinline__ void fence_proxy_async_smem() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}

// ---- warp-level tensor ops (bf16 m16n8k16, fp32 accumulate) --------------
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t& r0,
                                            uint32_t& r1, uint32_t& r2,
                                            uint32_t& r3) {
  asm volatile(
      "ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
      : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
      : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t& r0,
                                                  uint32_t& r1, uint32_t& r2,
                                                  uint32_t& r3) {
  asm volatile(
      "ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
      : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
      : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float (&c)[4],
                                               const uint32_t (&a)[4],
                                               uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 "
      "{%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ void named_bar_sync(int id, int nthreads) {
  asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(nthreads) : "memory");
}

#endif  // __CUDACC__

}  // namespace fk
