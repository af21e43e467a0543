// A sublayer's output as terms that whoever joins it to the stream sums (rows times numbers, routed experts' results gathered row by row), and the
// router that a launch runs on the rows it has just made: device code shared by the kernels that end a sublayer (streams.cu, norm_join.cu).
#pragma once

#include <math_constants.h>

#include "api.h"
#include "common.cuh"

namespace {

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
        const float f = o.factor[k] != nullptr ? o.scale[k] * o.factor[k][t] : o.scale[k];
#pragma unroll
        for (int i = 0; i < V; ++i) sum.v[i] = fmaf(f, y.v[i], sum.v[i]);
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

// ---------------------------------------------------------------- router
// The experts of rows t0 .. t0 + ROWS - 1 from their inputs h (in shared memory, ldh floats apart) by the whole block: the sums with a warp per three
// experts, all rows against every row of the matrix it reads, then a warp a row chooses.
// With `gate` the matrix has one more row behind the experts': the sigmoid of its product with row t goes to gate[t].
// smem, per row: z [n], c [n], best [groups], taken [groups] (int).
template <int ROWS, typename T>
__device__ __forceinline__ void route_rows(const lb_router& r, const float* h, int ldh, int width, int t0, int n_rows, float* smem) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5, n = r.n_experts, outputs = n + (r.gate != nullptr ? 1 : 0);
    const int per_row = 2 * n + 2 * r.groups;
    const T* R = static_cast<const T*>(r.matrix);
    for (int e0 = warp; e0 < outputs; e0 += 3 * n_warps) {
        float acc[3][ROWS];
        const T* w[3];
#pragma unroll
        for (int q = 0; q < 3; ++q) {
            w[q] = R + (size_t)min(e0 + q * n_warps, outputs - 1) * width;
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
                if (lane == 0 && e == n && e < outputs && t0 + i < n_rows) r.gate[t0 + i] = 1.0f / (1.0f + expf(-v));
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

inline size_t router_floats(const lb_router& r) { return 2 * (size_t)r.n_experts + 2 * (size_t)r.groups; }

inline int check_router(const lb_router& r) {
    LB_CHECK_ARG(r.n_experts > 0 && r.n_experts <= 4096 && r.top > 0 && r.ids != nullptr && r.weights != nullptr && r.groups >= 1 && r.keep >= 1 &&
                     r.keep <= r.groups && r.n_experts % r.groups == 0 && r.top <= r.n_experts / r.groups * r.keep,
                 "router: top %d of %d experts, %d of %d groups", r.top, r.n_experts, r.keep, r.groups);
    return LB_OK;
}

inline bool on16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
inline bool terms_on16(const lb_output_terms& o) {
    for (int k = 0; k < o.n_rows; ++k)
        if (o.ldy[k] % 4 != 0 || !on16(o.y[k])) return false;
    return o.pairs == nullptr || (o.ldp % 4 == 0 && on16(o.pairs) && (o.self == nullptr || (o.lds % 4 == 0 && on16(o.self))));
}
inline int check_terms(const lb_output_terms& o) {
    LB_CHECK_ARG(o.n_rows >= 0 && o.n_rows <= 4, "output terms: %d rows", o.n_rows);
    LB_CHECK_ARG(o.pairs == nullptr || (o.top > 0 && o.ids != nullptr), "output terms: gathered results need their experts");
    return LB_OK;
}

}  // namespace
