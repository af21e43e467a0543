// Where a sublayer between two norms meets the residual stream: x += norm_b(y), then the next sublayer's input h = norm_a(x), in one launch.
//
// y is the sum of the sublayer's output terms (row_terms.cuh), so the sum over routed experts and a gated shared expert need no launch of their own
// either; both norms are RMS norms over the whole row with 32-bit statistics.  Where the next sublayer routes its rows to experts, the same launch
// runs the router on h while the rows lie in shared memory.
//
// A block a row (four rows in turn where many rows are routed, so that a row of the router's matrix is read once for four).  A thread keeps its
// pieces of y, and then of the new x, in registers between the sums; gains and the old stream do not come from the kernel before this one and are
// asked for ahead of the wait for it.
#include "api.h"
#include "common.cuh"
#include "row_terms.cuh"

namespace {

// Sum over the block; `scratch` (two alternating halves of 32 floats) needs no barrier of its own between two calls.
__device__ __forceinline__ float block_total(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    v = lb_warp_sum(v);
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    return lb_warp_sum(lane < n_warps ? scratch[lane] : 0.0f);
}

// V values a piece, NV pieces a thread, ROWS rows a block one after the other.
template <int V, int NV, int ROWS, bool ROUTES, typename T>
__global__ void __launch_bounds__(512) norm_join_kernel(lb_norm_join_args a, lb_output_terms o, lb_router r, int n_rows) {
    extern __shared__ __align__(16) float smem[];       // with a router: the rows h, then the router's scratch
    __shared__ float sums[2][32];
    const int W = a.width, W4 = (W + 3) / 4 * 4, t0 = blockIdx.x * ROWS;
    constexpr bool kEarly = NV <= 2;
    Vals<V> gain[kEarly ? NV : 1], next_gain[kEarly ? NV : 1], x[NV];
    auto column = [&](int i) { return V * ((int)threadIdx.x + i * (int)blockDim.x); };
    auto gain_at = [&](const float* g, float offset, int c) {
        Vals<V> v;
        if (g != nullptr) v = load_vals<V>(g + c);
#pragma unroll
        for (int k = 0; k < V; ++k) v.v[k] = g != nullptr ? v.v[k] + offset : 1.0f;
        return v;
    };
    auto load_x = [&](int t) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (column(i) < W) x[i] = load_vals<V>(a.x + (size_t)t * a.ldx + column(i));
    };
    if constexpr (kEarly) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            if (column(i) >= W) break;
            gain[i] = gain_at(a.gain, a.gain_offset, column(i));
            if (a.h != nullptr) next_gain[i] = gain_at(a.next_gain, a.next_offset, column(i));
        }
    }
    load_x(t0);
    if (ROUTES && gridDim.x <= 64) {      // a few rows: the router's matrix starts on its way
        const char* R = static_cast<const char*>(r.matrix);
        const size_t bytes = (size_t)r.n_experts * W * sizeof(T);
        for (size_t i = (size_t)threadIdx.x * 128; i < bytes && i < 64 * 1024; i += (size_t)blockDim.x * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(R + i));
    }
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const float inv_w = 1.0f / (float)W;
    for (int t = t0; t < min(t0 + ROWS, n_rows); ++t) {
        if (t != t0) load_x(t);
        Vals<V> y[NV];
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            if (column(i) >= W) break;
            y[i] = terms_at<V, T>(o, t, column(i));
#pragma unroll
            for (int k = 0; k < V; ++k) ss = fmaf(y[i].v[k], y[i].v[k], ss);
        }
        const float f = a.scale / sqrtf(block_total(ss, sums[0]) * inv_w + a.eps);
        ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = column(i);
            if (c >= W) break;
            const Vals<V> g = kEarly ? gain[kEarly ? i : 0] : gain_at(a.gain, a.gain_offset, c);
#pragma unroll
            for (int k = 0; k < V; ++k) {
                x[i].v[k] = fmaf(y[i].v[k] * f, g.v[k], x[i].v[k]);
                ss = fmaf(x[i].v[k], x[i].v[k], ss);
            }
            store_vals<V>(a.x + (size_t)t * a.ldx + c, x[i]);
        }
        if (a.h == nullptr) {
            if (ROWS > 1) __syncthreads();      // the sums are used again
            continue;
        }
        const float n = 1.0f / sqrtf(block_total(ss, sums[1]) * inv_w + a.next_eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = column(i);
            if (c >= W) break;
            const Vals<V> g = kEarly ? next_gain[kEarly ? i : 0] : gain_at(a.next_gain, a.next_offset, c);
            Vals<V> h;
#pragma unroll
            for (int k = 0; k < V; ++k) h.v[k] = x[i].v[k] * n * g.v[k];
            store_vals<V>(static_cast<T*>(a.h) + (size_t)t * a.ldh + c, h);
            if (ROUTES) {
#pragma unroll
                for (int k = 0; k < V; ++k) smem[(t - t0) * W4 + c + k] = lb_to_float(lb_from_float<T>(h.v[k]));        // the router reads what the experts read
            }
        }
    }
    if constexpr (ROUTES) {
        __syncthreads();
        route_rows<ROWS, T>(r, smem, W4, W, t0, n_rows, smem + ROWS * W4);
    }
}

// Many rows of a single term without a router: a warp a row of up to 128 NV values, everything it reads asked for at once (which the choices inside a
// sum of terms do not let the compiler do), sums by shuffles, no block-wide barrier; the gains are read as they are used (the four rows of a block share
// them in the first-level cache).
template <int NV, typename T>
__global__ void __launch_bounds__(128) norm_join_warp_kernel(lb_norm_join_args a, lb_output_terms o, int n_rows) {
    const int lane = threadIdx.x & 31, t = blockIdx.x * 4 + (threadIdx.x >> 5), W = a.width;
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    if (t >= n_rows) return;
    Vals<4> x[NV], y[NV];
    float* xrow = a.x + (size_t)t * a.ldx;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * (lane + 32 * i);
        if (c >= W) break;
        x[i] = load_vals<4>(xrow + c);
        y[i] = load_vals<4>(o.y[0] + (size_t)t * o.ldy[0] + c);
    }
    const float times = o.factor[0] != nullptr ? o.scale[0] * o.factor[0][t] : o.scale[0];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        if (4 * (lane + 32 * i) >= W) break;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            y[i].v[k] *= times;
            ss = fmaf(y[i].v[k], y[i].v[k], ss);
        }
    }
    const float inv_w = 1.0f / (float)W, f = a.scale / sqrtf(lb_warp_sum(ss) * inv_w + a.eps);
    ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * (lane + 32 * i);
        if (c >= W) break;
        Vals<4> g;
        if (a.gain != nullptr) g = load_vals<4>(a.gain + c);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            x[i].v[k] = fmaf(y[i].v[k] * f, a.gain != nullptr ? g.v[k] + a.gain_offset : 1.0f, x[i].v[k]);
            ss = fmaf(x[i].v[k], x[i].v[k], ss);
        }
        store_vals<4>(xrow + c, x[i]);
    }
    if (a.h == nullptr) return;
    const float n = 1.0f / sqrtf(lb_warp_sum(ss) * inv_w + a.next_eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * (lane + 32 * i);
        if (c >= W) break;
        Vals<4> g, h;
        if (a.next_gain != nullptr) g = load_vals<4>(a.next_gain + c);
#pragma unroll
        for (int k = 0; k < 4; ++k) h.v[k] = x[i].v[k] * n * (a.next_gain != nullptr ? g.v[k] + a.next_offset : 1.0f);
        store_vals<4>(static_cast<T*>(a.h) + (size_t)t * a.ldh + c, h);
    }
}

template <int V, typename T>
int launch_norm_join(const lb_norm_join_args& a, const lb_output_terms& o, const lb_router& r, int n_rows, cudaStream_t s) {
    const bool routes = r.matrix != nullptr;
    const int pieces = a.width / V;
    if constexpr (V == 4) {
        if (!routes && o.n_rows == 1 && o.pairs == nullptr && n_rows > 296 && a.width <= 1024) {
            const dim3 grid((unsigned)((n_rows + 3) / 4)), block(128);
            if (a.width <= 256) LB_CHECK_CUDA(lb_launch_overlapped(norm_join_warp_kernel<2, T>, grid, block, 0, s, a, o, n_rows));
            else if (a.width <= 512) LB_CHECK_CUDA(lb_launch_overlapped(norm_join_warp_kernel<4, T>, grid, block, 0, s, a, o, n_rows));
            else if (a.width <= 768) LB_CHECK_CUDA(lb_launch_overlapped(norm_join_warp_kernel<6, T>, grid, block, 0, s, a, o, n_rows));
            else LB_CHECK_CUDA(lb_launch_overlapped(norm_join_warp_kernel<8, T>, grid, block, 0, s, a, o, n_rows));
            return LB_OK;
        }
    }
    const int rows = routes && n_rows > 148 && (size_t)4 * (a.width + 4 + router_floats(r)) * sizeof(float) <= 48 * 1024 ? 4 : 1;
    // Many rows: two pieces a thread, so that more rows are under way on an SM.
    int nv = n_rows > 296 && pieces > 64 ? 2 : 1;
    while ((pieces + nv - 1) / nv > 512) nv *= 2;
    nv = nv <= 2 ? nv : nv <= 4 ? 4 : 16;
    LB_CHECK_ARG((pieces + nv - 1) / nv <= 512, "norm join: rows of %d values are too long", a.width);
    int threads = ((pieces + nv - 1) / nv + 31) / 32 * 32;
    if (routes) threads = min(512, max(threads, 32 * max(rows, min(n_rows <= 148 ? 16 : 8, r.n_experts))));
    const size_t smem = routes ? rows * ((size_t)(a.width + 3) / 4 * 4 + router_floats(r)) * sizeof(float) : 0;
    LB_CHECK_ARG(smem <= 200 * 1024, "norm join: rows of %d values with a router do not fit shared memory", a.width);
    auto launch = [&](auto kernel) -> int {
        if (smem > 40 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, dim3((n_rows + rows - 1) / rows), dim3(threads), smem, s, a, o, r, n_rows));
        return LB_OK;
    };
#define LB_NORM_JOIN(NV)                                                          \
    return !routes     ? launch(norm_join_kernel<V, NV, 1, false, T>)             \
           : rows == 1 ? launch(norm_join_kernel<V, NV, 1, true, T>)              \
                       : launch(norm_join_kernel<V, NV, 4, true, T>)
    switch (nv) {
        case 1: LB_NORM_JOIN(1);
        case 2: LB_NORM_JOIN(2);
        case 4: LB_NORM_JOIN(4);
        default: LB_NORM_JOIN(16);
    }
#undef LB_NORM_JOIN
}

}  // namespace

extern "C" int lb_struct_bytes(int which) {
    switch (which) {
        case 0: return (int)sizeof(lb_output_terms);
        case 1: return (int)sizeof(lb_router);
        case 2: return (int)sizeof(lb_streams_args);
        case 3: return (int)sizeof(lb_norm_join_args);
        default: return 0;
    }
}

extern "C" int lb_norm_join(int dtype, const lb_norm_join_args* args, const lb_output_terms* terms, const lb_router* router, int n_rows, void* stream) {
    LB_CHECK_ARG(args != nullptr && terms != nullptr && args->x != nullptr && args->width > 0 && n_rows >= 0, "norm join: bad sizes");
    LB_CHECK_ARG(dtype == LB_F32 || dtype == LB_BF16, "norm join: unknown dtype %d", dtype);
    const lb_norm_join_args a = *args;
    const lb_output_terms o = *terms;
    lb_router r{};
    if (router != nullptr) r = *router;
    r.groups = r.matrix != nullptr ? r.groups : 1;
    if (int rc = check_terms(o)) return rc;
    LB_CHECK_ARG(o.n_rows > 0 || o.pairs != nullptr, "norm join: a sublayer's output has at least one term");
    LB_CHECK_ARG(r.matrix == nullptr || a.h != nullptr, "norm join: a router reads the next sublayer's input");
    if (r.matrix != nullptr)
        if (int rc = check_router(r)) return rc;
    if (n_rows == 0) return LB_OK;
    auto s = static_cast<cudaStream_t>(stream);
    const bool vec = a.width % 4 == 0 && a.ldx % 4 == 0 && on16(a.x) && on16(a.gain) && on16(a.next_gain) && (a.h == nullptr || (a.ldh % 4 == 0 && on16(a.h))) &&
                     terms_on16(o);
    if (dtype == LB_F32) return vec ? launch_norm_join<4, float>(a, o, r, n_rows, s) : launch_norm_join<1, float>(a, o, r, n_rows, s);
    return vec ? launch_norm_join<4, __nv_bfloat16>(a, o, r, n_rows, s) : launch_norm_join<1, __nv_bfloat16>(a, o, r, n_rows, s);
}
