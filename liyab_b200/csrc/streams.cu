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
#include "row_terms.cuh"

namespace {

constexpr int kMaxStreams = 16;

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
