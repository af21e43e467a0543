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

// Many rows of a single term: LANES threads a row of up to 4 LANES NV values, everything they read asked for at once (which the choices inside a sum of
// terms do not let the compiler do); `sum` adds up over them.  The rows of a block share the gains in the first-level cache.  A row that is not `live`
// takes part in the sums and writes nothing.  `kept` (or null): where the row h goes as floats for the router.
template <int NV, int LANES, typename T, typename Sum>
__device__ __forceinline__ void join_row(const lb_norm_join_args& a, const lb_output_terms& o, int t, int lane, bool live, float* kept, Sum sum) {
    const int W = a.width;
    Vals<4> x[NV], y[NV], g[NV];
    float* xrow = a.x + (size_t)t * a.ldx;
    const float* yrow = o.y[0] + (size_t)t * o.ldy[0];
    // Predicated, not skipped: a branch a piece would make every load wait for the one before.
    auto piece = [&](const float* p, int i, float otherwise) {
        Vals<4> v;
        const int c = 4 * (lane + LANES * i);
        const float4 q = c < W ? *reinterpret_cast<const float4*>(p + c) : make_float4(otherwise, otherwise, otherwise, otherwise);
        v.v[0] = q.x; v.v[1] = q.y; v.v[2] = q.z; v.v[3] = q.w;
        return v;
    };
#pragma unroll
    for (int i = 0; i < NV; ++i) y[i] = piece(yrow, i, 0.0f);
#pragma unroll
    for (int i = 0; i < NV; ++i) x[i] = piece(xrow, i, 0.0f);
    const float times = o.factor[0] != nullptr ? o.scale[0] * o.factor[0][t] : o.scale[0];
    const float gain_offset = a.gain != nullptr ? a.gain_offset : 1.0f, next_offset = a.next_gain != nullptr ? a.next_offset : 1.0f;
    auto gains = [&](const float* p) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            if (p != nullptr) g[i] = piece(p, i, 0.0f);
            else g[i].v[0] = g[i].v[1] = g[i].v[2] = g[i].v[3] = 0.0f;
        }
    };
    gains(a.gain);
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            y[i].v[k] *= times;
            ss = fmaf(y[i].v[k], y[i].v[k], ss);
        }
    const float inv_w = 1.0f / (float)W, f = a.scale / sqrtf(sum(ss) * inv_w + a.eps);
    ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            x[i].v[k] = fmaf(y[i].v[k] * f, g[i].v[k] + gain_offset, x[i].v[k]);
            ss = fmaf(x[i].v[k], x[i].v[k], ss);
        }
    if (a.h != nullptr) gains(a.next_gain);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * (lane + LANES * i);
        if (live && c < W) store_vals<4>(xrow + c, x[i]);
    }
    if (a.h == nullptr) return;
    const float n = 1.0f / sqrtf(sum(ss) * inv_w + a.next_eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * (lane + LANES * i);
        Vals<4> h;
#pragma unroll
        for (int k = 0; k < 4; ++k) h.v[k] = x[i].v[k] * n * (g[i].v[k] + next_offset);
        if (!live || c >= W) continue;
        if (kept != nullptr) {
            Vals<4> read;                   // the router reads what the experts read
#pragma unroll
            for (int k = 0; k < 4; ++k) read.v[k] = lb_to_float(lb_from_float<T>(h.v[k]));
            store_vals<4>(kept + c, read);
        }
        store_vals<4>(static_cast<T*>(a.h) + (size_t)t * a.ldh + c, h);
    }
}

template <int NV, typename T>
__global__ void __launch_bounds__(128) norm_join_warp_kernel(lb_norm_join_args a, lb_output_terms o, int n_rows) {
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    if (t < n_rows) join_row<NV, 32, T>(a, o, t, threadIdx.x & 31, true, nullptr, [](float v) { return lb_warp_sum(v); });
}

// The same with a router: 64 threads a row, four rows a block, then all of the block routes the four.
template <int NV, typename T>
__global__ void __launch_bounds__(256, 4) norm_join_routed_kernel(lb_norm_join_args a, lb_output_terms o, lb_router r, int n_rows) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float halves[2][8];
    const int warp = threadIdx.x >> 5, row = threadIdx.x >> 6, t0 = blockIdx.x * 4;
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    int turn = 0;
    join_row<NV, 64, T>(a, o, min(t0 + row, n_rows - 1), threadIdx.x & 63, t0 + row < n_rows, smem + row * a.width, [&](float v) {
        v = lb_warp_sum(v);
        float* both = halves[turn++];
        if ((threadIdx.x & 31) == 0) both[warp] = v;
        __syncthreads();
        return both[2 * row] + both[2 * row + 1];
    });
    __syncthreads();
    route_rows<4, T>(r, smem, a.width, a.width, t0, n_rows, smem + 4 * a.width);
}

template <int V, typename T>
int launch_norm_join(const lb_norm_join_args& a, const lb_output_terms& o, const lb_router& r, int n_rows, cudaStream_t s) {
    const bool routes = r.matrix != nullptr;
    const int pieces = a.width / V;
    if constexpr (V == 4) {
        const size_t scratch = routes ? 4 * (a.width + router_floats(r)) * sizeof(float) : 0;
        if (o.n_rows == 1 && o.pairs == nullptr && n_rows > 296 && a.width <= 1024 && scratch <= 48 * 1024) {
            const dim3 grid((unsigned)((n_rows + 3) / 4));
#define LB_JOIN_ROWS(NV)                                                                                                                   \
    if (routes) LB_CHECK_CUDA(lb_launch_overlapped(norm_join_routed_kernel<(NV + 1) / 2, T>, grid, dim3(256), scratch, s, a, o, r, n_rows)); \
    else LB_CHECK_CUDA(lb_launch_overlapped(norm_join_warp_kernel<NV, T>, grid, dim3(128), 0, s, a, o, n_rows))
            if (a.width <= 256) { LB_JOIN_ROWS(2); }
            else if (a.width <= 512) { LB_JOIN_ROWS(4); }
            else if (a.width <= 768) { LB_JOIN_ROWS(6); }
            else { LB_JOIN_ROWS(8); }
#undef LB_JOIN_ROWS
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
