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
// The same for results that are rounded to bfloat16: silu with the fast exponential and division; gelu by the rational
// approximation of the error function with five terms by C. Hastings (Abramowitz and Stegun, Handbook of Mathematical
// Functions, 7.1.26; absolute error at most 1.5e-7), erfc(y) = t (a1 + t (a2 + .. a5)) exp(-y^2), t = 1 / (1 + p y), y >= 0.
__device__ __forceinline__ float plain_act_fast(float v, int act) {
    if (act == ACT_GELU) {
        const float y = fabsf(v) * 0.70710678118654752f;
        const float t = __fdividef(1.0f, fmaf(0.3275911f, y, 1.0f));
        float a = fmaf(1.061405429f, t, -1.453152027f);
        a = fmaf(a, t, 1.421413741f);
        a = fmaf(a, t, -0.284496736f);
        a = fmaf(a, t, 0.254829592f);
        const float tail = 0.5f * a * t * __expf(-y * y);        // Phi(-|v|)
        return v * (v >= 0.0f ? 1.0f - tail : tail);
    }
    if (act == ACT_SILU) return __fdividef(v, 1.0f + __expf(-v));
    v = fmaxf(v, 0.0f);
    return v * v;
}
// N results at once: the choice outside the loop, the values' chains side by side
template <int N>
__device__ __forceinline__ void plain_acts_fast(float (&v)[N], int act) {
    if (act == ACT_GELU) {
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = plain_act_fast(v[j], ACT_GELU);
    } else if (act == ACT_SILU) {
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = plain_act_fast(v[j], ACT_SILU);
    } else {
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = plain_act_fast(v[j], ACT_RELU2);
    }
}
// 16 biases of consecutive features from f0 on (zeros without a bias or past the last feature)
__device__ __forceinline__ void load_bias16(const float* b, int f0, int features, float (&o)[16]) {
    if (b && f0 + 16 <= features && (((uintptr_t)(b + f0)) & 15) == 0) {
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
            const float4 v = __ldg((const float4*)(b + f0 + j));
            o[j] = v.x; o[j + 1] = v.y; o[j + 2] = v.z; o[j + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int j = 0; j < 16; ++j) o[j] = b && f0 + j < features ? b[f0 + j] : 0.0f;
    }
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
