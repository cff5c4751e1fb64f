// Kernels of attention whose heads are the difference of two score maps, and of experts whose weight meets their input.
//
// A stored head holds the two maps' keys side by side, D entries wide with map m in half m (zeros beyond the key's own
// size); the query of map m is zero outside half m.  Ordinary grouped-query attention with 2 H query heads and G
// key/value heads then gives both maps over the same values, which are stored once.
#include "api.h"
#include "common.cuh"

namespace dlmk {
namespace {

constexpr int HEAD_WARPS = 8;

template <int V> struct Lanes { float v[V]; };
template <int V> __device__ __forceinline__ Lanes<V> load_f32(const float* p) {
    Lanes<V> r;
    if constexpr (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else if constexpr (V == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        r.v[0] = x.x; r.v[1] = x.y;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V> __device__ __forceinline__ Lanes<V> load_act(const float* p) { return load_f32<V>(p); }
template <int V> __device__ __forceinline__ Lanes<V> load_act(const __nv_bfloat16* p) {
    Lanes<V> r;
    if constexpr (V == 1) {
        r.v[0] = __bfloat162float(*p);
    } else {
        uint32_t w[V / 2];
        if constexpr (V == 4) {
            const uint2 x = *reinterpret_cast<const uint2*>(p);
            w[0] = x.x; w[1] = x.y;
        } else {
            w[0] = *reinterpret_cast<const uint32_t*>(p);
        }
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
            r.v[2 * i] = __uint_as_float(w[i] << 16);
            r.v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_act(float* p, const Lanes<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(r.v[0], r.v[1]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void store_act(__nv_bfloat16* p, const Lanes<V>& r) {
    if constexpr (V == 1) {
        *p = __float2bfloat16_rn(r.v[0]);
    } else {
        uint32_t w[V / 2];
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(r.v[2 * i], r.v[2 * i + 1]);
            w[i] = *reinterpret_cast<const uint32_t*>(&b);
        }
        if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(w[0], w[1]);
        else *reinterpret_cast<uint32_t*>(p) = w[0];
    }
}

struct MapWriteParams {
    const float* proj; int ld;          // rows [q: H x 2 x d | k: G x 2 x d | v: G x dv | ...]
    const float* conv; int taps;        // [taps, C] (C = the channels of q, k and v), nullptr: no convolution
    float* state;                       // [slots, taps - 1, C]: the inputs before each request's next token, oldest first
    const int32_t* cu_q; const int32_t* token_req; const int32_t* state_slot;
    const float* qn; const float* kn; float eps;
    const int32_t* slots;
    void* q_out; void* k_cache; void* v_cache;
    int T, H, G, d, dv, D, page_size, total_pages, run;
    int* err;
};

// A warp takes one map of one query or key head, or one value head, and `run` tokens: the convolution over time, the
// norm over the map's d entries (not for values), the query into its half of q_out, key and value into the token's slot.
// Where a request brings a single token the warp also moves the carried inputs of its channels on: nobody else reads
// them in this launch.  NP groups of V neighbouring entries a lane; TAPS 0: any number of taps.
template <typename T, int V, int NP, int TAPS>
__global__ void __launch_bounds__(HEAD_WARPS * 32) map_norm_write_kernel(MapWriteParams p) {
    dep_wait();
    dep_launch_next();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int item = blockIdx.y * HEAD_WARPS + warp;
    const int nq = 2 * p.H, nk = 2 * p.G;
    if (item >= nq + nk + p.G) return;
    const bool is_q = item < nq, is_v = item >= nq + nk;
    const int width = is_v ? p.dv : p.d;
    const int c0 = is_v ? (nq + nk) * p.d + (item - nq - nk) * p.dv : item * p.d;
    const int C = (nq + nk) * p.d + p.G * p.dv;
    const int taps = p.conv == nullptr ? 1 : (TAPS > 0 ? TAPS : p.taps);
    const int keep = taps - 1;
    const int half = p.D / 2;
    const float* norm = is_q ? p.qn : p.kn;
    T* q_out = static_cast<T*>(p.q_out);
    T* kv = static_cast<T*>(is_v ? p.v_cache : p.k_cache);
    const int t_end = min(p.T, ((int)blockIdx.x + 1) * p.run);
    for (int t = blockIdx.x * p.run; t < t_end; ++t) {
        const int r = p.token_req[t];
        const int start = p.cu_q[r], n = p.cu_q[r + 1] - start;
        float* st = keep > 0 ? p.state + (long long)p.state_slot[r] * keep * C + c0 : nullptr;
        const float* x = p.proj + (long long)t * p.ld + c0;
        Lanes<V> y[NP];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int e = (i * 32 + lane) * V;
#pragma unroll
            for (int u = 0; u < V; ++u) y[i].v[u] = 0.f;
            if (e < width) {
                if (p.conv == nullptr) {
                    y[i] = load_f32<V>(x + e);
                } else {
                    auto add = [&](int j) {
                        const int back = keep - j;               // how many tokens before t
                        const Lanes<V> u = t - back >= start ? load_f32<V>(x - (long long)back * p.ld + e)
                                                             : load_f32<V>(st + (long long)(keep + (t - back - start)) * C + e);
                        const Lanes<V> w = load_f32<V>(p.conv + (long long)j * C + c0 + e);
#pragma unroll
                        for (int k = 0; k < V; ++k) y[i].v[k] = fmaf(w.v[k], u.v[k], y[i].v[k]);
                    };
                    if constexpr (TAPS > 0) {
#pragma unroll
                        for (int j = 0; j < TAPS; ++j) add(j);
                    } else {
                        for (int j = 0; j < taps; ++j) add(j);
                    }
                    if (n == 1 && keep > 0) {
                        for (int j = 0; j + 1 < keep; ++j) store_act<V>(st + (long long)j * C + e, load_f32<V>(st + (long long)(j + 1) * C + e));
                        store_act<V>(st + (long long)(keep - 1) * C + e, load_f32<V>(x + e));
                    }
                }
#pragma unroll
                for (int u = 0; u < V; ++u) ss = fmaf(y[i].v[u], y[i].v[u], ss);
            }
        }
        int slot = -1;
        if (!is_q) {
            slot = p.slots[t];
            if (slot >= p.total_pages * p.page_size) {
                if (lane == 0) *p.err = 2;
                slot = -1;
            }
            if (slot < 0) continue;
        }
        if (!is_v) {
            ss = warp_sum(ss);
            const float inv = 1.0f / sqrtf(ss / (float)p.d + p.eps);
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const int e = (i * 32 + lane) * V;
                if (e < width) {
                    const Lanes<V> w = load_f32<V>(norm + e);
#pragma unroll
                    for (int u = 0; u < V; ++u) y[i].v[u] = (y[i].v[u] * inv) * w.v[u];
                }
            }
        }
        // a map fills its half of the stored head, a value head all of it; entries beyond the own size are zeros
        const int span = is_v ? p.D : half;
        T* dst;
        if (is_q) {
            dst = q_out + ((long long)t * nq + item) * p.D;
        } else {
            const int g = is_v ? item - nq - nk : (item - nq) >> 1;
            dst = kv + (((long long)(slot / p.page_size) * p.G + g) * p.page_size + slot % p.page_size) * p.D;
        }
        const int at = is_v ? 0 : (item & 1) * half;                    // nq is even: the map's number for keys as well
        Lanes<V> zero;
#pragma unroll
        for (int u = 0; u < V; ++u) zero.v[u] = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int e = (i * 32 + lane) * V;
            if (e < span) {
                store_act<V>(dst + at + e, y[i]);
                if (is_q) store_act<V>(dst + (half - at) + e, zero);
            }
        }
    }
}

// out[t, h * dv + i] = c_i with a = o[t, 2h], b = o[t, 2h + 1] (D wide, the first dv entries count):
// c = (a - lambda b) / rms(a - lambda b) * factor * sigmoid(gate[t, h * dv + i]).  A warp a head of a token.
template <typename T, int V, int NP>
__global__ void __launch_bounds__(HEAD_WARPS * 32)
diff_norm_gate_kernel(const T* o, const float* gate, int ldg, T* out, long long heads, int H, int dv, int D, float lambda,
                      float eps, float factor) {
    dep_wait();
    dep_launch_next();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long i0 = (long long)blockIdx.x * HEAD_WARPS + warp;
    if (i0 >= heads) return;
    const long long t = i0 / H;
    const int h = (int)(i0 % H);
    const T* a = o + i0 * 2 * D;
    const float* g = gate != nullptr ? gate + t * ldg + (long long)h * dv : nullptr;
    Lanes<V> c[NP], z[NP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int e = (i * 32 + lane) * V;
        if (e < dv) {
            const Lanes<V> x = load_act<V>(a + e), y = load_act<V>(a + D + e);
            if (g != nullptr) z[i] = load_f32<V>(g + e);
#pragma unroll
            for (int u = 0; u < V; ++u) {
                c[i].v[u] = fmaf(-lambda, y.v[u], x.v[u]);
                ss = fmaf(c[i].v[u], c[i].v[u], ss);
            }
        }
    }
    ss = warp_sum(ss);
    const float inv = factor / sqrtf(ss / (float)dv + eps);
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int e = (i * 32 + lane) * V;
        if (e < dv) {
#pragma unroll
            for (int u = 0; u < V; ++u) c[i].v[u] *= g != nullptr ? inv / (1.0f + expf(-z[i].v[u])) : inv;
            store_act<V>(out + i0 * dv + e, c[i]);
        }
    }
}

// out[dest[t, j], :] = wts[t, j] * h[t, :]
template <typename T, int V>
__global__ void weigh_rows_kernel(const T* h, const float* wts, const int32_t* dest, T* out, int k, int H, int n, int* err) {
    dep_wait();
    dep_launch_next();
    const int pair = blockIdx.x;
    const int to = dest[pair];
    if (to < 0 || to >= n) {
        if (threadIdx.x == 0) *err = 4;
        return;
    }
    const float w = wts[pair];
    const T* src = h + (long long)(pair / k) * H;
    for (int e = threadIdx.x * V; e < H; e += blockDim.x * V) {
        Lanes<V> x = load_act<V>(src + e);
#pragma unroll
        for (int u = 0; u < V; ++u) x.v[u] *= w;
        store_act<V>(out + (long long)to * H + e, x);
    }
}

template <typename T, int V, int NP>
void launch_map_write(const MapWriteParams& p, dim3 grid, cudaStream_t stream) {
    const dim3 block(HEAD_WARPS * 32);
    if (p.conv != nullptr && p.taps == 3) launch_dep(map_norm_write_kernel<T, V, NP, 3>, grid, block, 0, stream, p);
    else if (p.conv != nullptr && p.taps == 4) launch_dep(map_norm_write_kernel<T, V, NP, 4>, grid, block, 0, stream, p);
    else launch_dep(map_norm_write_kernel<T, V, NP, 0>, grid, block, 0, stream, p);
}

template <typename T>
void map_write(const MapWriteParams& p, bool pairs, dim3 grid, cudaStream_t stream) {
    if (pairs) {
        if (p.D <= 64) launch_map_write<T, 2, 1>(p, grid, stream);
        else if (p.D <= 128) launch_map_write<T, 2, 2>(p, grid, stream);
        else launch_map_write<T, 2, 4>(p, grid, stream);
    } else {
        if (p.D <= 128) launch_map_write<T, 1, 4>(p, grid, stream);
        else launch_map_write<T, 1, 8>(p, grid, stream);
    }
}

template <typename T>
void diff_norm_gate_of(const void* o, const float* gate, int ldg, void* out, long long heads, int H, int dv, int D,
                       float lambda, float eps, float factor, bool quads, cudaStream_t stream) {
    const dim3 grid((unsigned)((heads + HEAD_WARPS - 1) / HEAD_WARPS)), block(HEAD_WARPS * 32);
#define DLM_DIFF(V, NP)                                                                                                \
    launch_dep(diff_norm_gate_kernel<T, V, NP>, grid, block, 0, stream, static_cast<const T*>(o), gate, ldg,          \
               static_cast<T*>(out), heads, H, dv, D, lambda, eps, factor)
    if (quads) { if (dv <= 128) DLM_DIFF(4, 1); else DLM_DIFF(4, 2); }
    else { if (dv <= 128) DLM_DIFF(1, 4); else DLM_DIFF(1, 8); }
#undef DLM_DIFF
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
bool aligned8(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 7) == 0; }

}  // namespace

void map_norm_write(const float* proj, int ld, const float* conv, int taps, float* state, const int32_t* cu_q,
                    const int32_t* token_req, const int32_t* state_slot, const float* qn, const float* kn, float eps,
                    const int32_t* slots, void* q_out, void* k_cache, void* v_cache, int T, int R, int num_single, int H,
                    int G, int d, int dv, int D, int page_size, int total_pages, int dtype, cudaStream_t stream) {
    if (T <= 0 || R <= 0) return;
    DLM_CHECK(D % 2 == 0 && D <= 256 && 2 * d <= D && dv <= D, "map_norm_write: a stored head (at most 256 wide) holds two keys or a value");
    DLM_CHECK(conv == nullptr || (taps >= 1 && taps <= 16), "map_norm_write: 1 to 16 taps");
    DLM_CHECK(conv == nullptr || taps == 1 || state != nullptr, "map_norm_write: a convolution over several tokens carries its inputs");
    const int items = 2 * H + 3 * G, gy = (items + HEAD_WARPS - 1) / HEAD_WARPS;
    // a token a warp until the machine is full several times over, then runs of tokens (they share the convolution's rows)
    long long run = (long long)T * gy / (8LL * sm_count());
    run = run < 1 ? 1 : (run > 8 ? 8 : run);
    MapWriteParams p{proj, ld, conv, taps, state, cu_q, token_req, state_slot, qn, kn, eps, slots, q_out, k_cache, v_cache,
                     T, H, G, d, dv, D, page_size, total_pages, (int)run, error_flag_ptr()};
    const dim3 grid((unsigned)((T + run - 1) / run), gy);
    const bool pairs = d % 2 == 0 && dv % 2 == 0 && D % 4 == 0 && ld % 2 == 0 && aligned8(proj) && aligned8(conv) &&
                       aligned8(state) && aligned8(qn) && aligned8(kn) && aligned8(q_out) && aligned8(k_cache) &&
                       aligned8(v_cache);
    if (dtype == F32) map_write<float>(p, pairs, grid, stream);
    else map_write<__nv_bfloat16>(p, pairs, grid, stream);
    check_launch("map_norm_write");
    if (conv != nullptr && taps > 1 && num_single < R)
        conv_state(proj, ld, state, cu_q, state_slot, R, 2 * (H + G) * d + G * dv, taps, 1, stream);
}

void diff_norm_gate(const void* o, const float* gate, int ldg, void* out, int T, int H, int dv, int D, float lambda,
                    float eps, float factor, int dtype, cudaStream_t stream) {
    if (T <= 0) return;
    DLM_CHECK(dv >= 1 && dv <= D && dv <= 256, "diff_norm_gate: values of 1 to 256 entries");
    const bool quads = dv % 4 == 0 && D % 4 == 0 && aligned16(o) && aligned16(out) &&
                       (gate == nullptr || (ldg % 4 == 0 && aligned16(gate)));
    const long long heads = (long long)T * H;
    if (dtype == F32) diff_norm_gate_of<float>(o, gate, ldg, out, heads, H, dv, D, lambda, eps, factor, quads, stream);
    else diff_norm_gate_of<__nv_bfloat16>(o, gate, ldg, out, heads, H, dv, D, lambda, eps, factor, quads, stream);
    check_launch("diff_norm_gate");
}

void weigh_rows(const void* h, const float* wts, const int32_t* dest, void* out, int T, int k, int H, int dtype,
                cudaStream_t stream) {
    if (T <= 0) return;
    const bool quads = H % 4 == 0 && aligned16(h) && aligned16(out);
    const dim3 grid(T * k), block(H >= 1024 ? 256 : 128);
    int* err = error_flag_ptr();
#define DLM_WEIGH(T_, V)                                                                                               \
    launch_dep(weigh_rows_kernel<T_, V>, grid, block, 0, stream, static_cast<const T_*>(h), wts, dest,                \
               static_cast<T_*>(out), k, H, T * k, err)
    if (dtype == F32) { if (quads) DLM_WEIGH(float, 4); else DLM_WEIGH(float, 1); }
    else { if (quads) DLM_WEIGH(__nv_bfloat16, 4); else DLM_WEIGH(__nv_bfloat16, 1); }
#undef DLM_WEIGH
    check_launch("weigh_rows");
}

}  // namespace dlmk
