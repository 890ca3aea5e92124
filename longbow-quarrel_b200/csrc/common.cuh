// Shared by every kernel file: dtype codes, conversions, error returns.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdlib.h>

#define LQ_F32 0
#define LQ_BF16 1

// Error codes returned by the extern "C" launchers (0 = launched).
#define LQ_OK 0
#define LQ_BAD_DTYPE -1
#define LQ_BAD_SIZE -2
#define LQ_NO_DRIVER -3

#define LQ_EXPORT extern "C" __attribute__((visibility("default")))

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

static inline int lq_launch_status() {
    cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? LQ_OK : (int)e;
}

// The first key that a row at position p sees under a mask given as one integer: w > 0, a sliding window of the
// last w positions; w < 0, the row's own block of -w positions (blocks are counted from the sequence's first
// position); 0, every earlier position.  It never decreases as p grows.
__device__ __forceinline__ int lq_first_key(int p, int w) {
    return w > 0 ? max(0, p - w + 1) : (w < 0 ? p - p % (-w) : 0);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// What a gated feed-forward makes of a gate and an up value: u g / (1 + e^(-g)) (limit 0), or with a limit m > 0 both are
// clamped first and the up value is shifted: (u + 1) g / (1 + e^(-1.702 g)), g = min(gate, m), u = clamp(up, -m, m).
struct Glu {
    float lim, slope, shift;
    __device__ __forceinline__ explicit Glu(float m)
        : lim(m > 0.f ? m : __builtin_huge_valf()), slope(m > 0.f ? 1.702f : 1.f), shift(m > 0.f ? 1.f : 0.f) {}
    template <bool FAST> __device__ __forceinline__ float of(float g, float u) const {
        g = fminf(g, lim);
        u = fminf(fmaxf(u, -lim), lim) + shift;
        return u * (g / (1.f + (FAST ? __expf(-slope * g) : expf(-slope * g))));
    }
};

// ------------------------------------------------------------------ programmatic dependent launch
// Kernels of a step follow one another on one stream.  Launched with launch_pdl, a kernel's
// blocks may be scheduled while the kernel before it is still draining; they run up to
// pdl_wait(), which returns once that kernel has completed and its writes are visible.  What a
// block does before pdl_wait() must not read anything an earlier kernel of the step writes, and
// must write nothing: index arithmetic, and prefetching of weights, which no kernel writes.
// pdl_launch_dependents() lets the kernel after this one be scheduled as early as possible.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

template <typename... KArgs, typename... Args>
static inline int launch_kernel(bool early, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    // LQ_PDL=0 in the environment launches every kernel strictly after the one before it.
    static const bool enabled = [] { const char* v = getenv("LQ_PDL"); return !(v && v[0] == '0'); }();
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = (enabled && early) ? 1 : 0;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
    return e == cudaSuccess ? LQ_OK : (int)e;
}

// A kernel whose blocks may be scheduled before the kernel ahead of it has finished.
template <typename... KArgs, typename... Args>
static inline int launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                             Args... args) {
    return launch_kernel(true, kernel, grid, block, smem, stream, args...);
}
// A kernel that starts only when the kernel ahead of it has finished: for kernels whose blocks
// fill an SM (their waiting blocks would keep the blocks of the kernel ahead off that SM).
template <typename... KArgs, typename... Args>
static inline int launch_after(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                               Args... args) {
    return launch_kernel(false, kernel, grid, block, smem, stream, args...);
}
