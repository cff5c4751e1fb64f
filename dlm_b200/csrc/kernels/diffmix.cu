// Kernels of attention whose heads are the difference of two score maps, and of experts whose weight meets their input.
//
// A stored head holds the two maps' keys side by side, D entries wide with map m in half m (zeros beyond the key's own
// size); the query of map m is zero outside half m.  Ordinary grouped-query attention with 2 H query heads and G
// key/value heads then gives both maps over the same values, which are stored once.
#include "api.h"
#include "common.cuh"
#include "lanes.cuh"

namespace dlmk {
namespace {

constexpr int HEAD_WARPS = 8;

struct MapWriteParams {
    const float* proj; int ld;          // rows [q: H x 2 x d | k: G x 2 x d | v: G x dv | ...]
    const float* conv; int taps;        // [taps, C] (C = the channels of q, k and v), nullptr: no convolution
    float* state;                       // [slots, taps - 1, C]: the inputs before each request's next token, oldest first
    const int32_t* cu_q; const int32_t* token_req; const int32_t* state_slot;
    const float* qn; const float* kn; float eps;
    const int32_t* slots;
    void* q_out; void* k_cache; void* v_cache;
    int T, H, G, d, dv, D, page_size, page_shift, total_pages;
    int* err;
};

// A warp takes one query or key head (both maps, side by side in the rows) or one value head, and RUN tokens: the
// convolution over time, a norm over each map's d entries (not for values), the two queries into their halves of q_out,
// key and value into the token's slot.  The rows of all its tokens (and of the taps - 1 before them) are asked for at once.
// Where a request brings a single token the warp also moves the carried inputs of its channels on: nobody else reads
// them in this launch.  NP groups of V neighbouring entries a lane (V divides d and dv, so that a group lies in one map);
// TAPS taps (1: no convolution over several tokens), 0: any number (read from the parameters, the rows then one by one).
template <typename T, int V, int NP, int TAPS, int RUN>
__global__ void __launch_bounds__(HEAD_WARPS * 32) map_norm_write_kernel(MapWriteParams p) {
    dep_wait();
    dep_launch_next();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int item = blockIdx.y * HEAD_WARPS + warp;
    if (item >= p.H + 2 * p.G) return;
    const bool is_q = item < p.H, is_v = item >= p.H + p.G;
    const int d = p.d, half = p.D / 2;
    const int width = is_v ? p.dv : 2 * d;
    const int c0 = is_v ? 2 * (p.H + p.G) * d + (item - p.H - p.G) * p.dv : item * 2 * d;
    const int C = 2 * (p.H + p.G) * d + p.G * p.dv;
    const int keep = (TAPS > 0 ? TAPS : p.taps) - 1;
    const float* conv = p.conv != nullptr ? p.conv + c0 : nullptr;
    const int t0 = blockIdx.x * RUN;
    const float* x0 = p.proj + (long long)t0 * p.ld + c0;               // the run's first row
    constexpr int LEAD = TAPS > 0 ? TAPS - 1 : 0;                       // rows in front of the run
    constexpr int ROWS = RUN + LEAD;
    Lanes<V> rows[ROWS][NP], w[TAPS > 0 ? TAPS : 1][NP], nw[NP];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int e = (i * 32 + lane) * V;
        const bool on = e < width;
#pragma unroll
        for (int a = 0; a < ROWS; ++a) {
            const int t = t0 + a - LEAD;
            if (on && t >= 0 && t < p.T) rows[a][i] = load_f32<V>(x0 + (a - LEAD) * p.ld + e);
        }
        if (on && TAPS > 0 && conv != nullptr) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j][i] = load_f32<V>(conv + j * C + e);
        }
        if (on && !is_v) nw[i] = load_f32<V>((is_q ? p.qn : p.kn) + (e < d ? e : e - d));
    }
    // the request of the run's first token; most runs lie in one request
    int r = p.token_req[t0], start = p.cu_q[r], count = p.cu_q[r + 1] - start;
    float* st = p.state + (long long)p.state_slot[r] * keep * C + c0;
    const int t_end = min(p.T, t0 + RUN);
    const bool same = p.token_req[t_end - 1] == r;
    const bool inside = same && t0 - keep >= start;                     // nobody needs a carried input
    Lanes<V> zero;
#pragma unroll
    for (int u = 0; u < V; ++u) zero.v[u] = 0.f;
#pragma unroll
    for (int a = 0; a < RUN; ++a) {
        const int t = t0 + a;
        if (t >= p.T) break;
        if (!same) {
            r = p.token_req[t];
            start = p.cu_q[r];
            count = p.cu_q[r + 1] - start;
            st = p.state + (long long)p.state_slot[r] * keep * C + c0;
        }
        Lanes<V> y[NP];
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int e = (i * 32 + lane) * V;
            y[i] = zero;
            if (e >= width) continue;
            if (conv == nullptr) {
                y[i] = rows[a + LEAD][i];
            } else if constexpr (TAPS > 0) {
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    Lanes<V> u = rows[a + j][i];                        // TAPS - 1 - j tokens before t
                    if (!inside && t - (TAPS - 1 - j) < start) u = load_f32<V>(st + (j + t - start) * C + e);
#pragma unroll
                    for (int k = 0; k < V; ++k) y[i].v[k] = fmaf(w[j][i].v[k], u.v[k], y[i].v[k]);
                }
            } else {
                for (int j = 0; j <= keep; ++j) {
                    const int back = keep - j;
                    const Lanes<V> u = t - back >= start ? load_f32<V>(x0 + (a - back) * p.ld + e)
                                                         : load_f32<V>(st + (j + t - start) * C + e);
                    const Lanes<V> wj = load_f32<V>(conv + j * C + e);
#pragma unroll
                    for (int k = 0; k < V; ++k) y[i].v[k] = fmaf(wj.v[k], u.v[k], y[i].v[k]);
                }
            }
            if (conv != nullptr && count == 1 && keep > 0) {
                for (int j = 0; j + 1 < keep; ++j) store_act<V>(st + j * C + e, load_f32<V>(st + (j + 1) * C + e));
                store_act<V>(st + (keep - 1) * C + e, rows[a + LEAD][i]);
            }
        }
        T* dst;
        if (is_q) {
            dst = static_cast<T*>(p.q_out) + ((long long)t * p.H + item) * 2 * p.D;
        } else {
            int slot = p.slots[t];
            if (slot >= p.total_pages * p.page_size) {
                if (lane == 0) *p.err = 2;
                slot = -1;
            }
            if (slot < 0) continue;
            const int page = p.page_shift >= 0 ? slot >> p.page_shift : slot / p.page_size;
            const int g = is_v ? item - p.H - p.G : item - p.H;
            dst = static_cast<T*>(is_v ? p.v_cache : p.k_cache) +
                  (((long long)page * p.G + g) * p.page_size + (slot - page * p.page_size)) * p.D;
        }
        if (is_v) {
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const int e = (i * 32 + lane) * V;
                if (e < width) store_act<V>(dst + e, y[i]);
            }
            for (int e = p.dv + lane; e < p.D; e += 32) dst[e] = from_f32<T>(0.f);
            continue;
        }
        float ss0 = 0.f, ss1 = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            float q = 0.f;
#pragma unroll
            for (int u = 0; u < V; ++u) q = fmaf(y[i].v[u], y[i].v[u], q);
            if ((i * 32 + lane) * V < d) ss0 += q; else ss1 += q;       // (beyond the head's own entries y is zero)
        }
        const float inv0 = 1.0f / sqrtf(warp_sum(ss0) / (float)d + p.eps);
        const float inv1 = 1.0f / sqrtf(warp_sum(ss1) / (float)d + p.eps);
        // map 1 goes to [0, d), map 2 to [half, half + d) of a key; of the two queries' rows likewise, with zeros in the
        // other map's place
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int e = (i * 32 + lane) * V;
            if (e >= width) continue;
            const bool second = e >= d;
            const int at = second ? half + e - d : e;
#pragma unroll
            for (int u = 0; u < V; ++u) y[i].v[u] = (y[i].v[u] * (second ? inv1 : inv0)) * nw[i].v[u];
            if (is_q) {
                store_act<V>(dst + (second ? p.D : 0) + at, y[i]);
                store_act<V>(dst + (second ? 0 : p.D) + at, zero);
            } else {
                store_act<V>(dst + at, y[i]);
            }
        }
        for (int e = d + lane; e < half; e += 32) {                     // where a half is wider than a map
            dst[e] = dst[half + e] = from_f32<T>(0.f);
            if (is_q) dst[p.D + e] = dst[p.D + half + e] = from_f32<T>(0.f);
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

template <typename T, int V, int NP, int RUN>
void launch_map_write(const MapWriteParams& p, int gy, cudaStream_t stream) {
    const dim3 grid((p.T + RUN - 1) / RUN, gy), block(HEAD_WARPS * 32);
    if (p.taps == 1) launch_dep(map_norm_write_kernel<T, V, NP, 1, RUN>, grid, block, 0, stream, p);
    else if (p.taps == 3) launch_dep(map_norm_write_kernel<T, V, NP, 3, RUN>, grid, block, 0, stream, p);
    else if (p.taps == 4) launch_dep(map_norm_write_kernel<T, V, NP, 4, RUN>, grid, block, 0, stream, p);
    else launch_dep(map_norm_write_kernel<T, V, NP, 0, RUN>, grid, block, 0, stream, p);
}

template <typename T>
void map_write(const MapWriteParams& p, int vec, int gy, cudaStream_t stream) {
    // a token a warp until the machine is full several times over, then four
    const bool many = (long long)p.T * gy > 16LL * sm_count();
#define DLM_MAP(V, NP)                                                                                                 \
    do { if (many) launch_map_write<T, V, NP, 4>(p, gy, stream); else launch_map_write<T, V, NP, 1>(p, gy, stream); } while (0)
    if (vec == 4) {
        if (p.D <= 128) DLM_MAP(4, 1);
        else DLM_MAP(4, 2);
    } else if (vec == 2) {
        if (p.D <= 64) DLM_MAP(2, 1);
        else if (p.D <= 128) DLM_MAP(2, 2);
        else DLM_MAP(2, 4);
    } else {
        if (p.D <= 128) DLM_MAP(1, 4);
        else DLM_MAP(1, 8);
    }
#undef DLM_MAP
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

}  // namespace

void map_norm_write(const float* proj, int ld, const float* conv, int taps, float* state, const int32_t* cu_q,
                    const int32_t* token_req, const int32_t* state_slot, const float* qn, const float* kn, float eps,
                    const int32_t* slots, void* q_out, void* k_cache, void* v_cache, int T, int R, int num_single, int H,
                    int G, int d, int dv, int D, int page_size, int total_pages, int dtype, cudaStream_t stream) {
    if (T <= 0 || R <= 0) return;
    DLM_CHECK(D % 2 == 0 && D <= 256 && 2 * d <= D && dv <= D, "map_norm_write: a stored head (at most 256 wide) holds two keys or a value");
    DLM_CHECK(conv == nullptr || (taps >= 1 && taps <= 16), "map_norm_write: 1 to 16 taps");
    DLM_CHECK(conv == nullptr || taps == 1 || state != nullptr, "map_norm_write: a convolution over several tokens carries its inputs");
    const int gy = (H + 2 * G + HEAD_WARPS - 1) / HEAD_WARPS;
    MapWriteParams p{proj, ld, conv, conv != nullptr ? taps : 1, state, cu_q, token_req, state_slot, qn, kn, eps, slots,
                     q_out, k_cache, v_cache, T, H, G, d, dv, D, page_size, -1, total_pages, error_flag_ptr()};
    if ((page_size & (page_size - 1)) == 0)
        for (p.page_shift = 0; (1 << p.page_shift) < page_size;) ++p.page_shift;
    // entries a lane takes side by side: as many as divide the sizes and the addresses allow
    auto fits = [&](int v) {
        const uintptr_t f32 = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(conv) |
                              reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(qn) | reinterpret_cast<uintptr_t>(kn);
        const uintptr_t act = reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache);
        return d % v == 0 && dv % v == 0 && D % (2 * v) == 0 && ld % v == 0 && f32 % (4 * v) == 0 && act % (4 * v) == 0;
    };
    const int vec = fits(4) ? 4 : (fits(2) ? 2 : 1);
    if (dtype == F32) map_write<float>(p, vec, gy, stream);
    else map_write<__nv_bfloat16>(p, vec, gy, stream);
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
