// Norms of layers that norm a sublayer's output: the centred norm with weight and bias alone, and the closing step of
// a sublayer (norm of its output, add to the residual, the next sublayer's input rounded from the new residual) in one
// pass over the rows.
//
// One block a row.  V > 0: the width is a multiple of four and a thread keeps V groups of four neighbouring entries in
// registers, so a row is read from memory once; V == 0: any width, the row is read again for every sum.  Mean and mean
// square deviation are two sums over the block in a fixed order (the second over the deviations themselves), so a row's
// result depends on the row and the width alone.  No kernel here waits on another.
#include "api.h"
#include "common.cuh"

namespace dlmk {
namespace {

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a);
    u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}

// ADD: resid[t] += norm(x[t]), out (may be nullptr) = the new resid[t], x zeroed when `clear`.  Otherwise
// out[i] = norm(x[rows ? rows[i] : i]).  CENTER: mean taken off, bias added; otherwise a root-mean-square norm.
template <typename T, bool ADD, bool CENTER, int V>
__global__ void post_norm_kernel(float* resid, float* x, const int32_t* rows, const float* __restrict__ w,
                                 const float* __restrict__ b, float eps, int clear, T* out, int H) {
    dep_wait();
    dep_launch_next();
    __shared__ float s_part[32];
    const long long dst = (long long)blockIdx.x * H;
    const long long src = (!ADD && rows != nullptr) ? (long long)rows[blockIdx.x] * H : dst;
    const float inv_h = 1.0f / (float)H;
    if constexpr (V > 0) {
        float4 v[V], r[V];
        float part = 0.f;
#pragma unroll
        for (int u = 0; u < V; ++u) {
            const int i = 4 * (threadIdx.x + u * blockDim.x);
            v[u] = i < H ? *reinterpret_cast<const float4*>(x + src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (ADD) r[u] = i < H ? *reinterpret_cast<const float4*>(resid + dst + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (CENTER) {
#pragma unroll
            for (int u = 0; u < V; ++u) part += (v[u].x + v[u].y) + (v[u].z + v[u].w);
            const float mean = block_sum(part, s_part) * inv_h;
#pragma unroll
            for (int u = 0; u < V; ++u)
                if (4 * (threadIdx.x + u * blockDim.x) < H) {
                    v[u].x -= mean; v[u].y -= mean; v[u].z -= mean; v[u].w -= mean;
                }
        }
        part = 0.f;
#pragma unroll
        for (int u = 0; u < V; ++u) {
            part = fmaf(v[u].x, v[u].x, part);
            part = fmaf(v[u].y, v[u].y, part);
            part = fmaf(v[u].z, v[u].z, part);
            part = fmaf(v[u].w, v[u].w, part);
        }
        const float inv = 1.0f / sqrtf(block_sum(part, s_part) * inv_h + eps);
#pragma unroll
        for (int u = 0; u < V; ++u) {
            const int i = 4 * (threadIdx.x + u * blockDim.x);
            if (i >= H) continue;
            const float4 ww = *reinterpret_cast<const float4*>(w + i);
            float4 n = make_float4(v[u].x * inv * ww.x, v[u].y * inv * ww.y, v[u].z * inv * ww.z, v[u].w * inv * ww.w);
            if (CENTER) {
                const float4 bb = *reinterpret_cast<const float4*>(b + i);
                n.x += bb.x; n.y += bb.y; n.z += bb.z; n.w += bb.w;
            }
            if (ADD) {
                n.x += r[u].x; n.y += r[u].y; n.z += r[u].z; n.w += r[u].w;
                store4(resid + dst + i, n);
                if (clear) store4(x + src + i, make_float4(0.f, 0.f, 0.f, 0.f));
            }
            if (!ADD || out != nullptr) store4(out + dst + i, n);
        }
    } else {
        float part = 0.f, mean = 0.f;
        if (CENTER) {
            for (int i = threadIdx.x; i < H; i += blockDim.x) part += x[src + i];
            mean = block_sum(part, s_part) * inv_h;
        }
        part = 0.f;
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            const float c = x[src + i] - mean;
            part = fmaf(c, c, part);
        }
        const float inv = 1.0f / sqrtf(block_sum(part, s_part) * inv_h + eps);
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            float n = (x[src + i] - mean) * inv * w[i];
            if (CENTER) n += b[i];
            if (ADD) {
                n += resid[dst + i];
                resid[dst + i] = n;
                if (clear) x[src + i] = 0.f;
            }
            if (!ADD || out != nullptr) out[dst + i] = from_f32<T>(n);
        }
    }
}

template <typename T, bool ADD, bool CENTER>
void launch_post_norm(float* resid, float* x, const int32_t* rows, const float* w, const float* b, float eps, int clear,
                      void* out, int n_rows, int H, cudaStream_t stream) {
    const uintptr_t all = reinterpret_cast<uintptr_t>(resid) | reinterpret_cast<uintptr_t>(x) |
                          reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(b) |
                          reinterpret_cast<uintptr_t>(out);
    const int quads = H / 4;
    T* o = static_cast<T*>(out);
    if (H % 4 == 0 && all % 16 == 0 && quads <= 8 * 256) {
        const int threads = quads >= 256 ? 256 : (quads + 31) / 32 * 32;
        const int v = (quads + threads - 1) / threads;
#define DLM_PN(V)                                                                                                    \
    launch_dep(post_norm_kernel<T, ADD, CENTER, V>, dim3(n_rows), dim3(threads), 0, stream, resid, x, rows, w, b, eps, \
               clear, o, H)
        if (v <= 1) DLM_PN(1);
        else if (v <= 2) DLM_PN(2);
        else if (v <= 4) DLM_PN(4);
        else DLM_PN(8);
#undef DLM_PN
        return;
    }
    launch_dep(post_norm_kernel<T, ADD, CENTER, 0>, dim3(n_rows), dim3(H >= 256 ? 256 : 128), 0, stream, resid, x, rows, w,
               b, eps, clear, o, H);
}

}  // namespace

void layer_norm(const float* x, const int32_t* rows, const float* w, const float* b, float eps, void* out, int n_rows,
                int H, int out_dtype, cudaStream_t stream) {
    if (n_rows <= 0) return;
    DLM_CHECK(H >= 1 && b != nullptr, "layer_norm: a width and a bias are needed");
    float* xx = const_cast<float*>(x);                      // only the adding form writes to its input
    if (out_dtype == F32)
        launch_post_norm<float, false, true>(nullptr, xx, rows, w, b, eps, 0, out, n_rows, H, stream);
    else
        launch_post_norm<__nv_bfloat16, false, true>(nullptr, xx, rows, w, b, eps, 0, out, n_rows, H, stream);
    check_launch("layer_norm");
}

void post_norm_add(float* resid, float* y, const float* w, const float* b, float eps, int centered, int clear, void* out,
                   int T, int H, int out_dtype, cudaStream_t stream) {
    if (T <= 0) return;
    DLM_CHECK(H >= 1 && (b != nullptr) == (centered != 0), "post_norm_add: the centred norm, and only it, has a bias");
    if (out_dtype == F32) {
        if (centered) launch_post_norm<float, true, true>(resid, y, nullptr, w, b, eps, clear, out, T, H, stream);
        else launch_post_norm<float, true, false>(resid, y, nullptr, w, b, eps, clear, out, T, H, stream);
    } else {
        if (centered) launch_post_norm<__nv_bfloat16, true, true>(resid, y, nullptr, w, b, eps, clear, out, T, H, stream);
        else launch_post_norm<__nv_bfloat16, true, false>(resid, y, nullptr, w, b, eps, clear, out, T, H, stream);
    }
    check_launch("post_norm_add");
}

}  // namespace dlmk
