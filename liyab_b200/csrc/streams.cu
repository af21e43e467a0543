// Blocks around several residual streams, and routers with corrected choices.
//
//   lb_streams_join     one launch between two sublayers.  The stream is a row of S parts of W values.  With y the sublayer's output (the sum of up
//                       to four terms, each a row times a number, or a row gathered from routed experts' results),
//                           X'[t] = sum_s M[s, t] X[s] + c[t] (scale * y)            (all t from the old X),
//                       then the next sublayer's input from the new parts, h = tanh(alpha sum_s a[s] X'[s]) gain + bias, and, where the next
//                       sublayer routes its rows to experts, the router on h.  Every step is optional: with `fresh` all parts start equal to
//                       a row of it; without a sublayer's output the parts stay as they are; with `rows` rows are gathered and nothing is written back.
//   lb_router_choice    the router by itself: z = R h (+ bias) in 32-bit, scores s = softmax(z) or sigmoid(z); the experts are chosen by
//                       s + correction among the `keep` best of `groups` equal groups of neighbours (a group counts as its best expert);
//                       weights = s of the chosen, times a factor, optionally over their sum.  Ties go to the lower index.
//   lb_terms_sum        x (+)= the sum of such terms, for arrangements with one stream.
//
// An expert's number of n_real or more stands for the identity: its result is the row `self` (the sublayer's input).
#include "api.h"
#include "common.cuh"

#include <math_constants.h>

namespace {

constexpr int kMaxStreams = 16;

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <>
__device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

// V values at a time: V = 4 (16-byte pieces) or 1.
template <int V>
struct Vals {
    float v[V];
};
template <int V, typename T>
__device__ __forceinline__ Vals<V> load_vals(const T* p) {
    Vals<V> r;
    if constexpr (V == 4) {
        const float4 f = load4<T>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = lb_to_float(*p);
    }
    return r;
}
template <int V>
__device__ __forceinline__ void store_vals(float* p, const Vals<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void store_vals(__nv_bfloat16* p, const Vals<V>& r) {
    if constexpr (V == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 u;
        u.x = *reinterpret_cast<const uint32_t*>(&lo);
        u.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

// Columns c .. c + V - 1 of row t of the terms' sum.
template <int V, typename T>
__device__ __forceinline__ Vals<V> terms_at(const lb_output_terms& o, int t, int c) {
    Vals<V> sum;
#pragma unroll
    for (int i = 0; i < V; ++i) sum.v[i] = 0.0f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        if (k >= o.n_rows) break;
        const Vals<V> y = load_vals<V>(o.y[k] + (size_t)t * o.ldy[k] + c);
#pragma unroll
        for (int i = 0; i < V; ++i) sum.v[i] = fmaf(o.scale[k], y.v[i], sum.v[i]);
    }
    if (o.pairs != nullptr) {
        // Two choices at a time: their experts, weights and places together, then their rows together.
        for (int k0 = 0; k0 < o.top; k0 += 2) {
            int e[2], at[2];
            float w[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int p = t * o.top + min(k0 + k, o.top - 1);
                e[k] = o.ids[p];
                w[k] = o.weights != nullptr ? o.weights[p] : 1.0f;
                at[k] = o.place != nullptr ? o.place[p] : p;
            }
            Vals<V> y[2];
#pragma unroll
            for (int k = 0; k < 2; ++k)
                if (k0 + k < o.top)
                    y[k] = e[k] < o.n_real ? load_vals<V>(o.pairs + (size_t)at[k] * o.ldp + c) : load_vals<V>(static_cast<const T*>(o.self) + (size_t)t * o.lds + c);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                if (k0 + k >= o.top) break;
#pragma unroll
                for (int i = 0; i < V; ++i) sum.v[i] = fmaf(w[k], y[k].v[i], sum.v[i]);
            }
        }
    }
    return sum;
}

template <int V, typename T>
__global__ void __launch_bounds__(256) terms_sum_kernel(lb_output_terms o, float* __restrict__ x, int64_t ldx, int n_rows, int width, int overwrite) {
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const long per_row = width / V, total = (long)n_rows * per_row;
    for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
        const int t = (int)(i / per_row), c = V * (int)(i - (long)t * per_row);
        Vals<V> s = terms_at<V, T>(o, t, c);
        float* dst = x + (size_t)t * ldx + c;
        if (!overwrite) {
            const Vals<V> old = load_vals<V>(dst);
#pragma unroll
            for (int k = 0; k < V; ++k) s.v[k] += old.v[k];
        }
        store_vals<V>(dst, s);
    }
}

// ---------------------------------------------------------------- router
// The experts of rows t0 .. t0 + ROWS - 1 from their inputs h (in shared memory, ldh floats apart) by the whole block: the sums with a warp per three
// experts, all rows against every row of the matrix it reads, then a warp a row chooses.
// smem, per row: z [n], c [n], best [groups], taken [groups] (int).
template <int ROWS, typename T>
__device__ __forceinline__ void route_rows(const lb_router& r, const float* h, int ldh, int width, int t0, int n_rows, float* smem) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5, n = r.n_experts;
    const int per_row = 2 * n + 2 * r.groups;
    const T* R = static_cast<const T*>(r.matrix);
    for (int e0 = warp; e0 < n; e0 += 3 * n_warps) {
        float acc[3][ROWS];
        const T* w[3];
#pragma unroll
        for (int q = 0; q < 3; ++q) {
            w[q] = R + (size_t)min(e0 + q * n_warps, n - 1) * width;
#pragma unroll
            for (int i = 0; i < ROWS; ++i) acc[q][i] = 0.0f;
        }
        if (width % 4 == 0 && (reinterpret_cast<uintptr_t>(R) & 15) == 0) {        // four values a lane and load
            for (int k0 = 4 * lane; k0 < width; k0 += 4 * 64) {
                float4 b[3][2];
#pragma unroll
                for (int u = 0; u < 2; ++u)
#pragma unroll
                    for (int q = 0; q < 3; ++q) b[q][u] = k0 + 128 * u < width ? load4<T>(w[q] + k0 + 128 * u) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                for (int i = 0; i < ROWS; ++i)
#pragma unroll
                    for (int u = 0; u < 2; ++u) {
                        if (k0 + 128 * u >= width) break;
                        const float4 a = load4<float>(h + (size_t)i * ldh + k0 + 128 * u);
#pragma unroll
                        for (int q = 0; q < 3; ++q) acc[q][i] = fmaf(a.x, b[q][u].x, fmaf(a.y, b[q][u].y, fmaf(a.z, b[q][u].z, fmaf(a.w, b[q][u].w, acc[q][i]))));
                    }
            }
        } else {
            for (int k = lane; k < width; k += 32)
#pragma unroll
                for (int q = 0; q < 3; ++q)
#pragma unroll
                    for (int i = 0; i < ROWS; ++i) acc[q][i] = fmaf(h[(size_t)i * ldh + k], lb_to_float(w[q][k]), acc[q][i]);
        }
#pragma unroll
        for (int q = 0; q < 3; ++q)
#pragma unroll
            for (int i = 0; i < ROWS; ++i) {
                const int e = e0 + q * n_warps;
                const float v = lb_warp_sum(acc[q][i]);
                if (lane == 0 && e < n) smem[i * per_row + e] = r.bias != nullptr ? v + r.bias[e] : v;
            }
    }
    __syncthreads();
    const int t = t0 + warp;
    if (warp >= ROWS || t >= n_rows) return;
    float* z = smem + warp * per_row;
    float* c = z + n;
    float* best = c + n;
    int* taken = reinterpret_cast<int*>(best + r.groups);
    float top_z = -CUDART_INF_F, sum = 0.0f;
    if (r.softmax) {
        for (int e = lane; e < n; e += 32) top_z = fmaxf(top_z, z[e]);
        top_z = lb_warp_max(top_z);
        for (int e = lane; e < n; e += 32) sum += expf(z[e] - top_z);
        sum = lb_warp_sum(sum);
    }
    for (int e = lane; e < n; e += 32) {
        const float s = r.softmax ? expf(z[e] - top_z) / sum : 1.0f / (1.0f + expf(-z[e]));
        z[e] = s;
        c[e] = r.correction != nullptr ? s + r.correction[e] : s;
    }
    __syncwarp();
    // The largest of v[0 .. count), the lowest index among equals; every lane gets the index.  Floats compare as unsigned numbers in this form.
    auto argmax = [&](const float* v, int count) {
        unsigned key = 0;
        int at = 0x7fffffff;
        for (int i = lane; i < count; i += 32) {
            const unsigned bits = __float_as_uint(v[i]), k = bits & 0x80000000u ? ~bits : bits | 0x80000000u;
            if (at == 0x7fffffff || k > key) { key = k; at = i; }
        }
        const unsigned top_key = __reduce_max_sync(0xffffffffu, key);
        return min((int)__reduce_min_sync(0xffffffffu, key == top_key ? (unsigned)at : 0x7fffffffu), count - 1);
    };
    if (r.groups > 1 && r.keep < r.groups) {
        const int size = n / r.groups;
        for (int g = lane; g < r.groups; g += 32) {
            float m = -CUDART_INF_F;
            for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, c[e]);
            best[g] = m;
            taken[g] = 0;
        }
        __syncwarp();
        for (int k = 0; k < r.keep; ++k) {
            const int g = argmax(best, r.groups);
            __syncwarp();
            if (lane == 0) { taken[g] = 1; best[g] = -CUDART_INF_F; }
            __syncwarp();
        }
        for (int e = lane; e < n; e += 32)
            if (!taken[e / size]) c[e] = -CUDART_INF_F;
        __syncwarp();
    }
    float total = 0.0f;
    for (int k = 0; k < r.top; ++k) {
        const int e = argmax(c, n);
        const float s = z[e];
        total += s;
        __syncwarp();
        if (lane == 0) c[e] = -CUDART_INF_F;
        __syncwarp();
        if (lane == 0) {
            r.ids[(size_t)t * r.top + k] = e;
            r.weights[(size_t)t * r.top + k] = r.renormalise != 0 ? s : s * r.scale;
        }
    }
    if (r.renormalise != 0 && lane == 0)
        for (int k = 0; k < r.top; ++k) r.weights[(size_t)t * r.top + k] *= r.scale / total;
}

template <typename T>
__global__ void __launch_bounds__(512) router_choice_kernel(lb_router r, const T* __restrict__ h, int64_t ldh, int width) {
    extern __shared__ __align__(16) float smem[];
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const int t = blockIdx.x;
    for (int c = threadIdx.x; c < width; c += blockDim.x) smem[c] = lb_to_float(h[(size_t)t * ldh + c]);
    __syncthreads();
    route_rows<1, T>(r, smem, 0, width, t, t + 1, smem + (width + 3) / 4 * 4);
}

// ---------------------------------------------------------------- the streams between two sublayers
// A block per ROWS rows.  MAXS: as many streams as a thread keeps (EXACT: S is MAXS); ROUTES: with a router.
template <int V, int MAXS, bool EXACT, int ROWS, bool ROUTES, typename T>
__global__ void __launch_bounds__(512) streams_join_kernel(lb_streams_args a, lb_output_terms o, lb_router r, int n_rows) {
    extern __shared__ __align__(16) float smem[];       // with a router: the rows h, then the router's scratch
    __shared__ float hc[kMaxStreams * kMaxStreams + 2 * kMaxStreams];
    const int S = EXACT ? MAXS : a.n_streams, W = a.width;
    float* mix = hc;
    float* to = hc + S * S;
    float* next = to + S;
    // Weights: read before the wait for the kernel before this one.
    const bool moves = o.n_rows > 0 || o.pairs != nullptr, goes_on = a.h != nullptr;
    if (moves)
        for (int i = threadIdx.x; i < S * S + S; i += blockDim.x) hc[i] = i < S * S ? a.mix[i] : a.to[i - S * S];
    if (goes_on)
        for (int i = threadIdx.x; i < S; i += blockDim.x) next[i] = a.next_in != nullptr ? a.next_in[i] : 1.0f;
    const float alpha = a.alpha != nullptr ? a.alpha[0] : 1.0f;
    const int t0 = blockIdx.x * ROWS, c_first = V * threadIdx.x;
    // The thread's first columns of the old streams too, where a sublayer's output joins them: the launch that wrote them lies before that sublayer's.
    Vals<V> x_early[EXACT ? MAXS : 1], g_early, gain_early, offset_early;
    const bool early = EXACT && ROWS == 1 && moves && c_first < W;
    if (early) {
#pragma unroll
        for (int s = 0; s < (EXACT ? MAXS : 1); ++s) x_early[s] = load_vals<V>(a.x + (size_t)t0 * a.ldx + (size_t)s * W + c_first);
        if (a.scale != nullptr) g_early = load_vals<V>(a.scale + c_first);
        if (goes_on && a.alpha != nullptr) {
            gain_early = load_vals<V>(a.gain + c_first);
            offset_early = load_vals<V>(a.offset + c_first);
        }
    }
    if (ROUTES && gridDim.x <= 64) {      // a few rows: the router's matrix starts on its way
        const char* R = static_cast<const char*>(r.matrix);
        const size_t bytes = (size_t)r.n_experts * W * sizeof(T);
        for (size_t i = (size_t)threadIdx.x * 128; i < bytes && i < 64 * 1024; i += (size_t)blockDim.x * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(R + i));
    }
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    __syncthreads();
    const int W4 = (W + 3) / 4 * 4;
    for (int t = t0; t < min(t0 + ROWS, n_rows); ++t) {
        float* xrow = a.x + (size_t)(a.rows != nullptr ? a.rows[t] : t) * a.ldx;
        for (int c = c_first; c < W; c += V * blockDim.x) {
            Vals<V> x[MAXS];
            const bool have = early && c == c_first;
            if (have) {
#pragma unroll
                for (int s = 0; s < (EXACT ? MAXS : 1); ++s) x[s] = x_early[s];
            } else if (a.fresh != nullptr) {
                x[0] = load_vals<V>(a.fresh + (size_t)t * a.ldf + c);
#pragma unroll
                for (int s = 1; s < MAXS; ++s) x[s] = x[0];
            } else {
#pragma unroll
                for (int s = 0; s < MAXS; ++s)
                    if (EXACT || s < S) x[s] = load_vals<V>(xrow + (size_t)s * W + c);
            }
            Vals<V> u;
#pragma unroll
            for (int i = 0; i < V; ++i) u.v[i] = 0.0f;
            if (moves) {
                Vals<V> y = terms_at<V, T>(o, t, c);
                if (a.scale != nullptr) {
                    const Vals<V> g = have ? g_early : load_vals<V>(a.scale + c);
#pragma unroll
                    for (int i = 0; i < V; ++i) y.v[i] *= g.v[i];
                }
#pragma unroll(EXACT ? MAXS : 1)
                for (int q = 0; q < S; ++q) {
                    Vals<V> z;
#pragma unroll
                    for (int i = 0; i < V; ++i) z.v[i] = to[q] * y.v[i];
#pragma unroll
                    for (int s = 0; s < MAXS; ++s) {
                        if (!EXACT && s >= S) break;
                        const float m = mix[s * S + q];
#pragma unroll
                        for (int i = 0; i < V; ++i) z.v[i] = fmaf(m, x[s].v[i], z.v[i]);
                    }
                    store_vals<V>(xrow + (size_t)q * W + c, z);
                    if (goes_on) {
                        const float n = next[q];
#pragma unroll
                        for (int i = 0; i < V; ++i) u.v[i] = fmaf(n, z.v[i], u.v[i]);
                    }
                }
            } else {
#pragma unroll
                for (int q = 0; q < MAXS; ++q) {
                    if (!EXACT && q >= S) break;
                    if (a.fresh != nullptr) store_vals<V>(xrow + (size_t)q * W + c, x[q]);
                    if (goes_on) {
                        const float n = next[q];
#pragma unroll
                        for (int i = 0; i < V; ++i) u.v[i] = fmaf(n, x[q].v[i], u.v[i]);
                    }
                }
            }
            if (!goes_on) continue;
            if (a.alpha != nullptr) {
                const Vals<V> g = have ? gain_early : load_vals<V>(a.gain + c), b = have ? offset_early : load_vals<V>(a.offset + c);
#pragma unroll
                for (int i = 0; i < V; ++i) u.v[i] = fmaf(tanhf(alpha * u.v[i]), g.v[i], b.v[i]);
            }
            store_vals<V>(static_cast<T*>(a.h) + (size_t)t * a.ldh + c, u);
            if (ROUTES) {
#pragma unroll
                for (int i = 0; i < V; ++i) smem[(t - t0) * W4 + c + i] = lb_to_float(lb_from_float<T>(u.v[i]));        // the router reads what the experts read
            }
        }
    }
    if constexpr (ROUTES) {
        __syncthreads();
        route_rows<ROWS, T>(r, smem, W4, W, t0, n_rows, smem + ROWS * W4);
    }
}

size_t router_floats(const lb_router& r) { return 2 * (size_t)r.n_experts + 2 * (size_t)r.groups; }

int check_router(const lb_router& r) {
    LB_CHECK_ARG(r.n_experts > 0 && r.n_experts <= 4096 && r.top > 0 && r.ids != nullptr && r.weights != nullptr && r.groups >= 1 && r.keep >= 1 &&
                     r.keep <= r.groups && r.n_experts % r.groups == 0 && r.top <= r.n_experts / r.groups * r.keep,
                 "router: top %d of %d experts, %d of %d groups", r.top, r.n_experts, r.keep, r.groups);
    return LB_OK;
}

bool on16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
bool terms_on16(const lb_output_terms& o) {
    for (int k = 0; k < o.n_rows; ++k)
        if (o.ldy[k] % 4 != 0 || !on16(o.y[k])) return false;
    return o.pairs == nullptr || (o.ldp % 4 == 0 && on16(o.pairs) && (o.self == nullptr || (o.lds % 4 == 0 && on16(o.self))));
}
int check_terms(const lb_output_terms& o) {
    LB_CHECK_ARG(o.n_rows >= 0 && o.n_rows <= 4, "output terms: %d rows", o.n_rows);
    LB_CHECK_ARG(o.pairs == nullptr || (o.top > 0 && o.ids != nullptr), "output terms: gathered results need their experts");
    return LB_OK;
}

template <int V, typename T>
int launch_join(const lb_streams_args& a, const lb_output_terms& o, const lb_router& r, int n_rows, cudaStream_t s) {
    const int pieces = a.width / V;
    // Steps of many rows route four rows a block: they share what the block reads of the router's matrix, and four warps choose at once.
    const int rows = r.matrix != nullptr && n_rows > 148 && (size_t)4 * (a.width + router_floats(r)) * sizeof(float) <= 48 * 1024 ? 4 : 1;
    int threads = min(512, max(32, (pieces + 31) / 32 * 32));
    if (r.matrix != nullptr) threads = max(threads, 32 * max(rows, min(n_rows <= 148 ? 16 : 8, r.n_experts)));
    const size_t smem = r.matrix != nullptr ? rows * ((size_t)(a.width + 3) / 4 * 4 + router_floats(r)) * sizeof(float) : 0;
    LB_CHECK_ARG(smem <= 200 * 1024, "streams: rows of %d values with a router do not fit shared memory", a.width);
    auto launch = [&](auto kernel) -> int {
        if (smem > 40 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, dim3((n_rows + rows - 1) / rows), dim3(threads), smem, s, a, o, r, n_rows));
        return LB_OK;
    };
#define LB_JOIN(MAXS, EXACT)                                                                    \
    return r.matrix == nullptr ? launch(streams_join_kernel<V, MAXS, EXACT, 1, false, T>)       \
           : rows == 1         ? launch(streams_join_kernel<V, MAXS, EXACT, 1, true, T>)        \
                               : launch(streams_join_kernel<V, MAXS, EXACT, 4, true, T>)
    if constexpr (V == 1) {
        if (a.n_streams <= 4) LB_JOIN(4, false);
        LB_JOIN(kMaxStreams, false);
    } else {
        switch (a.n_streams) {
            case 1: LB_JOIN(1, true);
            case 2: LB_JOIN(2, true);
            case 3: LB_JOIN(3, true);
            case 4: LB_JOIN(4, true);
            default:
                if (a.n_streams <= 8) LB_JOIN(8, false);
                LB_JOIN(kMaxStreams, false);
        }
    }
#undef LB_JOIN
}

}  // namespace

extern "C" int lb_streams_join(int dtype, const lb_streams_args* args, const lb_output_terms* terms, const lb_router* router, int n_rows, void* stream) {
    LB_CHECK_ARG(args != nullptr && args->n_streams >= 1 && args->n_streams <= kMaxStreams && args->width > 0 && n_rows >= 0 && args->x != nullptr,
                 "streams: %d streams (1 to %d)", args == nullptr ? 0 : args->n_streams, kMaxStreams);
    LB_CHECK_ARG(dtype == LB_F32 || dtype == LB_BF16, "streams: unknown dtype %d", dtype);
    const lb_streams_args a = *args;
    lb_output_terms o{};
    lb_router r{};
    if (terms != nullptr) o = *terms;
    if (router != nullptr) r = *router;
    r.groups = r.matrix != nullptr ? r.groups : 1;
    if (int rc = check_terms(o)) return rc;
    const bool moves = o.n_rows > 0 || o.pairs != nullptr;
    LB_CHECK_ARG(!moves || (a.mix != nullptr && a.to != nullptr && a.rows == nullptr && a.fresh == nullptr), "streams: a sublayer's output needs its mixing weights and every row in place");
    LB_CHECK_ARG(a.alpha == nullptr || (a.gain != nullptr && a.offset != nullptr), "streams: the norm needs gain and offset");
    LB_CHECK_ARG(r.matrix == nullptr || a.h != nullptr, "streams: a router reads the next sublayer's input");
    if (r.matrix != nullptr)
        if (int rc = check_router(r)) return rc;
    if (n_rows == 0) return LB_OK;
    auto s = static_cast<cudaStream_t>(stream);
    const bool vec = a.width % 4 == 0 && a.ldx % 4 == 0 && on16(a.x) && (a.fresh == nullptr || (a.ldf % 4 == 0 && on16(a.fresh))) && on16(a.scale) && on16(a.gain) &&
                     on16(a.offset) && (a.h == nullptr || (a.ldh % 4 == 0 && on16(a.h))) && terms_on16(o);
    if (dtype == LB_F32) return vec ? launch_join<4, float>(a, o, r, n_rows, s) : launch_join<1, float>(a, o, r, n_rows, s);
    return vec ? launch_join<4, __nv_bfloat16>(a, o, r, n_rows, s) : launch_join<1, __nv_bfloat16>(a, o, r, n_rows, s);
}

extern "C" int lb_router_choice(int dtype, const lb_router* router, const void* h, int64_t ldh, int n_rows, int width, void* stream) {
    LB_CHECK_ARG(router != nullptr && router->matrix != nullptr && n_rows >= 0 && width > 0, "router: bad sizes");
    if (int rc = check_router(*router)) return rc;
    if (n_rows == 0) return LB_OK;
    auto s = static_cast<cudaStream_t>(stream);
    const int threads = 32 * max(1, min(16, router->n_experts));
    const size_t smem = ((size_t)(width + 3) / 4 * 4 + router_floats(*router)) * sizeof(float);
    LB_CHECK_ARG(smem <= 200 * 1024, "router: rows of %d values do not fit shared memory", width);
    auto launch = [&](auto kernel, auto* rows) -> int {
        if (smem > 48 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, dim3(n_rows), dim3(threads), smem, s, *router, rows, ldh, width));
        return LB_OK;
    };
    if (dtype == LB_F32) return launch(router_choice_kernel<float>, static_cast<const float*>(h));
    if (dtype == LB_BF16) return launch(router_choice_kernel<__nv_bfloat16>, static_cast<const __nv_bfloat16*>(h));
    return lb_fail(LB_ERR_INVALID_ARGUMENT, "router: unknown dtype %d", dtype);
}

extern "C" int lb_terms_sum(int dtype, const lb_output_terms* terms, float* x, int64_t ldx, int n_rows, int width, int overwrite, void* stream) {
    LB_CHECK_ARG(terms != nullptr && n_rows >= 0 && width > 0, "sum of output terms: bad sizes");
    LB_CHECK_ARG(dtype == LB_F32 || dtype == LB_BF16, "sum of output terms: unknown dtype %d", dtype);
    if (int rc = check_terms(*terms)) return rc;
    if (n_rows == 0) return LB_OK;
    const lb_output_terms o = *terms;
    auto s = static_cast<cudaStream_t>(stream);
    const bool vec = width % 4 == 0 && ldx % 4 == 0 && on16(x) && terms_on16(o);
    const long total = (long)n_rows * (width / (vec ? 4 : 1));
    const dim3 grid((unsigned)min((total + 255) / 256, (long)148 * 16));
    if (dtype == LB_F32) {
        if (vec) LB_CHECK_CUDA(lb_launch_overlapped(terms_sum_kernel<4, float>, grid, dim3(256), 0, s, o, x, ldx, n_rows, width, overwrite));
        else LB_CHECK_CUDA(lb_launch_overlapped(terms_sum_kernel<1, float>, grid, dim3(256), 0, s, o, x, ldx, n_rows, width, overwrite));
    } else {
        if (vec) LB_CHECK_CUDA(lb_launch_overlapped(terms_sum_kernel<4, __nv_bfloat16>, grid, dim3(256), 0, s, o, x, ldx, n_rows, width, overwrite));
        else LB_CHECK_CUDA(lb_launch_overlapped(terms_sum_kernel<1, __nv_bfloat16>, grid, dim3(256), 0, s, o, x, ldx, n_rows, width, overwrite));
    }
    return LB_OK;
}
