// Shared helpers of the sm_100a kernels: element types, conversions, error reporting.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>
#include <stdio.h>
#include <string.h>

// Element type codes used across the C interface.
#define BRAID_F32 0
#define BRAID_BF16 1

// Error codes returned by every entry point: 0 is success, a positive value is a
// cudaError_t, a negative value is a refusal by the entry point itself whose text
// braid_last_error() returns.
#define BRAID_OK 0
#define BRAID_REFUSED (-1)

#ifdef __cplusplus
extern "C" {
#endif
const char* braid_last_error(void);
#ifdef __cplusplus
}
#endif

void braid_set_error(const char* fmt, ...);

#define BRAID_REFUSE(...)            \
    do {                             \
        braid_set_error(__VA_ARGS__); \
        return BRAID_REFUSED;        \
    } while (0)

#define BRAID_LAUNCH_CHECK()                         \
    do {                                             \
        cudaError_t e__ = cudaGetLastError();        \
        if (e__ != cudaSuccess) {                    \
            braid_set_error("%s:%d: %s", __FILE__, __LINE__, cudaGetErrorString(e__)); \
            return (int)e__;                         \
        }                                            \
        return BRAID_OK;                             \
    } while (0)

// Programmatic dependent launch.  Every kernel of the library is launched with the
// attribute that lets it begin while its predecessor in the stream drains, calls
// pdl_trigger() at its top (so that its own successor may be scheduled early; later where a kernel says why) and
// pdl_wait() before its first access to memory that an earlier kernel may have written
// (or may still read).  What comes before pdl_wait() must touch only weights and the
// kernel's own shared or tensor memory.  BRAIDINFER_PDL=0 in the environment turns the
// attribute off; the two instructions are then no-ops.
int braid_pdl_enabled(void);

__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

template <typename... KArgs, typename... Args>
static inline cudaError_t braid_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                       cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = braid_pdl_enabled();
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Activations of the gated feed-forwards, out = act(gate) * up.  An entry point that takes an epilogue
// `mode` takes the activation's code in bits 4..7 of it (0: silu).
#define BRAID_ACT_SILU 0
#define BRAID_ACT_GELU_TANH 1
#define BRAID_ACT_COUNT 2
// gelu in its tanh form, 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))) = z * sigmoid(2 u), u the tanh's argument
__device__ __forceinline__ float gelu_tanh_f32(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return 0.5f * z * (1.f + tanhf(u));
}
__device__ __forceinline__ float silu_f32(float z) { return z / (1.f + expf(-z)); }
// The clamped gated unit: g = min(gate, limit), u = clamp(up, -limit, limit); g * sigmoid(alpha * g) * (u + 1).
__device__ __forceinline__ float glu_clamp_f32(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}
__device__ __forceinline__ float glu_act(float g, int act) {
    return act == BRAID_ACT_GELU_TANH ? gelu_tanh_f32(g) : silu_f32(g);
}
// The same with the fast exponential and division: a few ulp, far inside the bfloat16 rounding of the
// result, and no slow path for the infinities that the exponential reaches (g / inf = 0 is the right limit).
__device__ __forceinline__ float glu_act_fast(float g, int act) {
    const float e = act == BRAID_ACT_GELU_TANH ? -1.5957691216057308f * (g + 0.044715f * g * g * g) : -g;
    return __fdividef(g, 1.f + __expf(e));
}

// V neighbouring numbers as float32, V = 1 or as many as 16 bytes hold (p on 16 bytes then).
template <typename T, int V>
__device__ __forceinline__ void load_run(const T* p, float* v) {
    if constexpr (V == 1) {
        v[0] = to_f32(p[0]);
    } else {
        __align__(16) T raw[V];
        *reinterpret_cast<uint4*>(raw) = *reinterpret_cast<const uint4*>(p);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = to_f32(raw[e]);
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_run(T* p, const float* v) {
    if constexpr (V == 1) {
        p[0] = from_f32<T>(v[0]);
    } else {
        __align__(16) T raw[V];
#pragma unroll
        for (int e = 0; e < V; ++e) raw[e] = from_f32<T>(v[e]);
        *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(raw);
    }
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

// Sum over a block of up to 1024 threads, same order every time; all threads get the result.
__device__ __forceinline__ float block_sum(float v, float* smem32) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) smem32[warp] = v;
    __syncthreads();
    const int nw = (blockDim.x + 31) >> 5;
    float t = (lane < nw) ? smem32[lane] : 0.f;
    t = warp_sum(t);
    return t;
}
