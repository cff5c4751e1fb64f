// Shared device helpers: element conversion, warp/block reductions, error checks.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cstdint>
#include <stdexcept>
#include <string>
#include <utility>

namespace dlmk {

enum DType : int { F32 = 0, BF16 = 1 };

#define DLM_CHECK(cond, msg)                                                        \
    do {                                                                            \
        if (!(cond)) throw std::invalid_argument(std::string("dlm_b200 kernels: ") + (msg)); \
    } while (0)

inline void check_launch(const char* what) {
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess)
        throw std::runtime_error(std::string("dlm_b200 kernels: launch of ") + what + " failed: " +
                                 cudaGetErrorString(e));
}

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

// Sum over a block in a fixed order (per-thread partials -> warp trees -> serial over warps).
// `scratch` holds at least 32 floats.  Every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nwarp; ++i) t += scratch[i];
    return t;
}

// Programmatic dependent launch.  A kernel launched through launch_dep() may be made resident
// while the kernel before it in the stream is still running, as soon as every block of that kernel
// has called dep_launch_next() or ended.  It must call dep_wait() before it reads anything an earlier
// kernel wrote and before it writes anything at all; dep_wait() returns when the earlier kernel
// has ended and its writes are visible.  Every block calls dep_wait() before it ends, so that
// "this kernel has ended" implies "all earlier kernels have ended".  What a kernel does before
// dep_wait() (index arithmetic, loads of weights, which no kernel writes) overlaps the end of the
// kernel before it.  Launched in the ordinary way both calls do nothing.  Pointers to what earlier
// kernels write (and to what this kernel writes) are not declared __restrict__ in such kernels:
// the compiler may move an access through a __restrict__ pointer across dep_wait(), which is an
// assembly statement that clobbers memory and so orders every other access.
__device__ __forceinline__ void dep_launch_next() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void dep_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

// Whether launch_dep() asks for the early launch (off: DLM_B200_NO_PDL=1, or set_dep_launch(false)).
bool dep_launch_enabled();
void set_dep_launch(bool on);

template <typename... P, typename... A>
inline void launch_dep(void (*kernel)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, A&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = dep_launch_enabled() ? 1 : 0;
    cudaLaunchKernelEx(&cfg, kernel, std::forward<A>(args)...);   // an error shows in check_launch()
}

// Multiprocessors of the current device (asked once).
int sm_count();

// Device pointer of the host-mapped error flag (see take_error_flag in api.h).
int* error_flag_ptr();

// silu(z) = z / (1 + exp(-z)), as the reference writes it
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// gelu(z) = z (1 + erf(z / sqrt 2)) / 2, the exact form
__device__ __forceinline__ float gelu_exact_f(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f)); }
// gelu(z) = z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) / 2, the tanh form
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
}
// What a storing epilogue does to acc (+ bias) before it rounds: gelu for EPI (an Epilogue of api.h) == 3, EPI_GELU,
// its tanh form for 4, EPI_GELU_TANH; nothing otherwise.
template <int EPI> __device__ __forceinline__ float epi_act(float v) {
    return EPI == 3 ? gelu_exact_f(v) : (EPI == 4 ? gelu_tanh_f(v) : v);
}
// The gated epilogues, 2 (EPI_SWIGLU), 5 (EPI_GEGLU_TANH) and 6 (EPI_CLAMP_GLU): what the gate half goes through before it meets the up
// half.  glu_act_fast: for results that are rounded to bfloat16 (fast exponential and division; the tanh form of gelu
// is z times the logistic function of twice the tanh's argument).
constexpr bool epi_is_glu(int epi) { return epi == 2 || epi == 5 || epi == 6; }
// whether the `bias` of a product is something the epilogue may read (a bias, or the constants of EPI_CLAMP_GLU)
constexpr bool epi_takes_bias(int epi) { return epi == 0 || epi == 3 || epi == 4 || epi == 6; }
template <int EPI> __device__ __forceinline__ float glu_act(float g) { return EPI == 5 ? gelu_tanh_f(g) : silu_f(g); }
template <int EPI> __device__ __forceinline__ float glu_act_fast(float g) {
    const float z = EPI == 5 ? 1.59576912160573071176f * (g + 0.044715f * g * g * g) : g;
    return __fdividef(g, 1.0f + __expf(-z));
}
// One output of a gated epilogue from its gate and up sums; `c`: the constants of EPI_CLAMP_GLU {limit, alpha, shift}.
template <int EPI, bool FAST> __device__ __forceinline__ float glu_out(float g, float u, const float* c) {
    if (EPI == 6) {
        const float limit = c[0], z = fminf(g, limit), v = fminf(fmaxf(u, -limit), limit) + c[2];
        return (FAST ? __fdividef(z, 1.0f + __expf(-c[1] * z)) : z / (1.0f + expf(-c[1] * z))) * v;
    }
    return (FAST ? glu_act_fast<EPI>(g) : glu_act<EPI>(g)) * u;
}

}  // namespace dlmk
