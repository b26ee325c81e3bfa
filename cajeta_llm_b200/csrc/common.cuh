// Shared helpers of the hand-written sm_100a kernels.
//
// Every exported function has C linkage, takes raw device pointers plus a stream,
// launches asynchronously and returns 0 or a negative "refused" code / positive
// cudaError_t.  Storage types are passed as small integer codes so that one entry
// point serves the 32-bit path and the bfloat16 path.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdlib.h>
#include <string.h>

#define CJ_F32 0
#define CJ_BF16 1

// refusal codes (negative so they never collide with cudaError_t)
#define CJ_ERR_DTYPE (-2)     // dtype combination not instantiated
#define CJ_ERR_SIZE (-3)      // a size this kernel does not take
#define CJ_ERR_ALIGN (-4)     // pointer or stride alignment this kernel needs
#define CJ_ERR_ARG (-5)       // null pointer or negative count

#define CJ_EXPORT extern "C" __attribute__((visibility("default")))

namespace cj {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

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

// x / (1 + exp(-x)), the reference's SiLU (model/Prim.cajeta:1822-1847)
__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }

// The gate of a gated feed-forward, from its two products g (gate) and u (up).  limit == 0:
// g * sigmoid(alpha g + cubic g^3) * u, which is silu(g) * u for (1, 0) and, because
// (1 + tanh y) / 2 = sigmoid(2 y), the tanh form of gelu for (2 sqrt(2 / pi), 2 sqrt(2 / pi) 0.044715).
// limit > 0, the capped form: g = min(g, limit), u = clamp(u, -limit, limit), g * sigmoid(alpha g) * (u + 1).
__device__ __forceinline__ float gated_act(float g, float u, float limit, float alpha, float cubic) {
    if (limit > 0.0f) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
    }
    return g / (1.0f + expf(-g * (alpha + cubic * g * g))) * u;
}
// the same with the fast exponential and division, for results that are rounded to bfloat16
__device__ __forceinline__ float gated_act_fast(float g, float u, float limit, float alpha, float cubic) {
    if (limit > 0.0f) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return __fdividef(g, 1.0f + __expf(-alpha * g)) * (u + 1.0f);
    }
    return __fdividef(g, 1.0f + __expf(-g * (alpha + cubic * g * g))) * u;
}

// The activation of a product's result: max(v, 0)^2, v Phi(v) (gelu by the error function) or silu
constexpr int ACT_NONE = 0, ACT_RELU2 = 1, ACT_GELU = 2, ACT_SILU = 3;
__device__ __forceinline__ float plain_act(float v, int act) {
    if (act == ACT_GELU) return 0.5f * v * (1.0f + erff(v * 0.70710678118654752f));
    if (act == ACT_SILU) return silu(v);
    v = fmaxf(v, 0.0f);
    return v * v;
}

// Launches overlap their neighbours in the stream (programmatic dependent launch): a kernel
// may be set up on the SMs while the one before it is still draining.  Every kernel of this
// library therefore begins with after_predecessor(), which returns once all earlier work in
// the stream is complete and visible - before it nothing that another kernel writes may be
// read and nothing it reads may be written - and release_successor(), which lets the next
// kernel's blocks be scheduled as SM resources free up (they wait at their own
// after_predecessor()).  In a kernel launched the ordinary way both are no-ops.
__device__ __forceinline__ void after_predecessor() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void release_successor() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// CAJETA_B200_SERIAL_LAUNCH=1 turns the overlap off (every kernel then starts after the one before has ended), and so
// does cj_set_launch_overlap(0), which the engine calls for a model whose plan asks for plain stream order.
// CAJETA_B200_SERIAL_LIBS=name,name turns it off for the kernels of the named libraries alone (a library names itself
// with CJ_LIB before it includes this header): a way to find which neighbours' overlap a fault depends on.
#ifndef CJ_LIB
#define CJ_LIB "?"
#endif
static int g_launch_overlap = -1;      // -1: not asked yet; one copy a library
inline bool overlap_launches() {
    if (g_launch_overlap < 0) {
        const char* e = getenv("CAJETA_B200_SERIAL_LAUNCH");
        g_launch_overlap = (e && e[0] == '1') ? 0 : 1;
        const char* libs = getenv("CAJETA_B200_SERIAL_LIBS");
        const size_t n = strlen(CJ_LIB);
        for (const char* at = libs ? strstr(libs, CJ_LIB) : nullptr; at; at = strstr(at + 1, CJ_LIB))      // whole names only
            if ((at == libs || at[-1] == ',') && (at[n] == ',' || at[n] == 0)) g_launch_overlap = 0;
    }
    return g_launch_overlap != 0;
}

template <typename... P, typename... A>
inline void launch(void (*kernel)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, A&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = overlap_launches() ? 1 : 0;
    cudaLaunchKernelEx(&cfg, kernel, static_cast<A&&>(args)...);      // an error is left for launch_status()
}

// The same launch in plain stream order: the kernel starts when everything before it in the stream has ended.  For a
// kernel that holds most of an SM for long (a successor set up beside it would only take room from its own later blocks);
// such a kernel does not call release_successor() either, so what follows it starts when it has ended.
template <typename... P, typename... A>
inline void launch_in_order(void (*kernel)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, A&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cfg.numAttrs = 0;
    cudaLaunchKernelEx(&cfg, kernel, static_cast<A&&>(args)...);
}

inline int launch_status() {
    cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? 0 : (int)e;
}

}  // namespace cj

// 0: this library's kernels launch in plain stream order from now on; 1: they may overlap their neighbours again
// (unless the environment turned the overlap off)
CJ_EXPORT void cj_set_launch_overlap(int on) {
    if (!on) cj::g_launch_overlap = 0;
    else { cj::g_launch_overlap = -1; cj::overlap_launches(); }
}
