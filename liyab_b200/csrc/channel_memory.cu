// Mixers whose memory is a matrix per head with a decay per key channel:
//     S_t = diag(a_t) S_{t-1} + k_t u_t^T,      o_t = S_t^T q_t,
// with u_t = v_t (gated linear attention) or, under the delta rule, u_t = beta_t (v_t - (diag(a_t) S_{t-1})^T k_t), so that what is written
// replaces what the decayed memory already answers to the key.  S is dim x vdim, 32-bit, zero at a sequence's start.
//
// Around the recurrence, all from the float rows of one projection [q | k | v | ..]:
//   queries, keys and values may pass a causal convolution per channel over `taps` inputs and SiLU; queries and keys may be made unit vectors
//   per head; queries carry a factor; n_head / kv_head heads in a row share one query and one key row;
//   the decays come through a map of low rank, z = A2 (the projection's columns a_off ..) + bias: log a = log sigmoid(z) / tau, or
//   log a = -exp(a_log[head]) softplus(z);
//   every head's o is divided by its root mean square, times a gain, times sigmoid or silu of a gate, whose pre-activations are columns
//   of the projection or come through a map of low rank as well.
//
// State of a request: [head][dim][vdim] floats (S), behind them the convolution's ring [taps][channels]: the input of position p lies in entry
// p mod taps, so a row reads entries that no other row of a step of single tokens writes.
//
// Two forms.  lb_channel_memory_rows: one launch does everything from the projection to the gated heads, a block per (request, head), rows one
// after the other: decode steps and short portions.  lb_channel_memory_pieces: every piece of 32 rows of every request a block of its own.  With
// b_t[d] the sum of log a[d] from the piece's start to row t, inside a piece
//     P(t, j) = sum_d q_t[d] k_j[d] exp(b_t[d] - b_j[d]) for j <= t,      A(t, j) the same with k_t for q_t and j < t;
//     without the delta rule u_j = v_j;  with it, (I + diag(beta) A) U = diag(beta) (V - K~ S0), K~_t = exp(b_t) k_t, S0 the state before the piece,
//     so U = M V - (M K~) S0 with M = (I + diag(beta) A)^-1 diag(beta), a triangular solve of the piece alone;
//     o_t = S0^T (exp(b_t) q_t) + sum_{j <= t} P(t, j) u_j,      S1 = diag(exp(b_n)) S0 + sum_j (exp(b_n - b_j) k_j) u_j^T.
// Every exponent is at most 0 (the pairs' exponentials are made pair by pair), so a strong decay underflows to zero and nothing overflows.
// Pairs of a row of a piece's second half with a key of its first meet at the border between them (two factors, each at most 1).
// Launches: the pieces' own matrices (convolution, unit vectors and decays included), the scan over a request's pieces, the outputs with norm and gate.
#include "api.h"
#include "common.cuh"

#include <math_constants.h>

namespace {

constexpr int kPiece = 32;

__device__ __forceinline__ float cm_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float cm_gate(float z, int act) { return act == LB_GATE_SILU ? z * cm_sigmoid(z) : cm_sigmoid(z); }
// The logarithm (base 2) of a channel's decay from its pre-activation.
__device__ __forceinline__ float cm_log2_decay(const lb_channel_memory& m, float z, int h) {
    const float l = m.a_log != nullptr ? -expf(m.a_log[h]) * lb_softplus(z) : -lb_softplus(-z) / m.tau;
    return l * kLbLog2e;
}

__device__ __forceinline__ void cm_cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cm_cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cm_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cm_cp_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
// Asks for `count` floats (all threads of the block together).
__device__ __forceinline__ void cm_fetch(float* dst, const float* src, int count) {
    if (((reinterpret_cast<uintptr_t>(src) | (uint32_t)__cvta_generic_to_shared(dst)) & 15) == 0 && (count & 3) == 0) {
        for (int i = threadIdx.x; i < count / 4; i += blockDim.x) cm_cp_async16(dst + 4 * i, src + 4 * i);
    } else {
        for (int i = threadIdx.x; i < count; i += blockDim.x) cm_cp_async4(dst + i, src + i);
    }
}

// A row of a low-rank map: sum_r w[r] x[r].  Ranks that split into 16-byte pieces are read in those, four pieces at a time in flight.
template <typename T>
__device__ __forceinline__ float low_rank(const T* __restrict__ w, const float* __restrict__ x, int rank) {
    constexpr int N = 16 / sizeof(T);
    float acc[2] = {0.0f, 0.0f};
    if (rank % N == 0 && ((reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(x)) & 15) == 0) {
        for (int r0 = 0; r0 < rank; r0 += 4 * N) {
            uint4 wv[4];
            float4 xv[4][N / 4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int r = min(r0 + u * N, rank - N);
                wv[u] = *reinterpret_cast<const uint4*>(w + r);
#pragma unroll
                for (int k = 0; k < N / 4; ++k) xv[u][k] = *reinterpret_cast<const float4*>(x + r + 4 * k);
            }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                if (r0 + u * N >= rank) break;
                const T* wt = reinterpret_cast<const T*>(&wv[u]);
                const float* xt = reinterpret_cast<const float*>(xv[u]);
#pragma unroll
                for (int k = 0; k < N; ++k) acc[k & 1] = fmaf(lb_to_float(wt[k]), xt[k], acc[k & 1]);
            }
        }
        return acc[0] + acc[1];
    }
    for (int r = 0; r < rank; ++r) acc[0] = fmaf(lb_to_float(w[r]), x[r], acc[0]);
    return acc[0];
}

struct StepArgs {
    const float* proj;         // [T, ld]
    int64_t ld;
    const int32_t* positions;  // [T]
    const int32_t* tok_seq;    // [T]
    const int32_t* q_start;    // [S + 1]
    const int32_t* slots;      // [S]
    float* state;
    float* o;                  // [T, ldo] the heads before norm and gate, or null
    int64_t ldo;
    void* heads;               // [T, ldh]
    int64_t ldh;
};

__device__ __forceinline__ int channels_of(const lb_channel_memory& m) { return 2 * m.kv_head * m.dim + m.n_head * m.vdim; }

// Channel c of row `row` of a request that starts at row0 (position pos): the convolution over its inputs with SiLU, or the input as it is.
__device__ __forceinline__ float conv_channel(const lb_channel_memory& m, const StepArgs& a, const float* ring, int c, int row, int row0, int pos, int channels) {
    if (m.conv == nullptr) return a.proj[(size_t)row * a.ld + c];
    const int K = m.taps;
    const float* w = m.conv + (size_t)c * K;
    auto input = [&](int back) -> float {              // the input `back` tokens ago
        if (row - back >= row0) return a.proj[(size_t)(row - back) * a.ld + c];
        return pos - back >= 0 ? ring[(size_t)((pos - back) % K) * channels + c] : 0.0f;
    };
    float acc = 0.0f;
    if (K <= 4) {                                      // all inputs and taps asked for together
        float u[4], t[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            u[k] = k < K ? input(k) : 0.0f;
            t[k] = k < K ? w[K - 1 - k] : 0.0f;
        }
        acc = fmaf(t[0], u[0], fmaf(t[1], u[1], fmaf(t[2], u[2], t[3] * u[3])));
    } else {
        for (int k = K - 1; k >= 0; --k) acc = fmaf(w[K - 1 - k], input(k), acc);
    }
    return acc * cm_sigmoid(acc);
}

// ---------------------------------------------------------------- row by row, from the projection to the gated heads
// Thread (c, ds) owns rows ds, ds + DS, .. of column c of the head's S (in shared memory where it fits, else where it lies).  The state travels
// before this kernel waits for the one before it.
template <typename T>
__global__ void __launch_bounds__(512) channel_memory_rows_kernel(lb_channel_memory m, StepArgs a, int ep2, int staged, int write_ring) {
    extern __shared__ __align__(16) float smem[];
    const int seq = blockIdx.x, h = blockIdx.y, D = m.dim, E = m.vdim, share = m.n_head / m.kv_head;
    const int row0 = a.q_start[seq], row1 = a.q_start[seq + 1];
    const int channels = channels_of(m);
    float* slot = a.state + (size_t)a.slots[seq] * m.slot_stride;
    float* st = slot + (size_t)h * D * E;
    float* ring = slot + (size_t)m.n_head * D * E;
    float* qs = smem;                          // [D]
    float* ks = qs + D;                        // [D]
    float* keep = ks + D;                      // [D]
    float* vs = keep + D;                      // [E]
    float* gate = vs + E;                      // [E]
    float* os = gate + E;                      // [E]
    float* red = os + E;                       // [threads]
    float* S = staged ? smem + (3 * (D + E) + blockDim.x + 3) / 4 * 4 : st;
    if (staged && row1 > row0) {
        cm_fetch(S, st, D * E);
        cm_cp_commit();
    }
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    if (row1 <= row0) return;
    const int c = threadIdx.x & (ep2 - 1), ds = threadIdx.x / ep2, DS = blockDim.x / ep2, lane = threadIdx.x & 31;
    const bool live = c < E;
    const int g = h / share;                   // the query and key row of the head
    for (int row = row0; row < row1; ++row) {
        const int pos = a.positions[row];
        const float* pr = a.proj + (size_t)row * a.ld;
        // The row's queries, keys, values, decays and gates: one value a thread and trip, so that the maps' weights and the inputs travel together.
        for (int i = threadIdx.x; i < 3 * D + 2 * E; i += blockDim.x) {
            if (i < D) {
                const int d = i;
                const T* w = static_cast<const T*>(m.a2) + ((size_t)h * D + d) * m.rank;
                const float z = low_rank(w, pr + m.a_off, m.rank) + (m.z_bias != nullptr ? m.z_bias[h * D + d] : 0.0f);
                keep[d] = exp2f(cm_log2_decay(m, z, h));
            } else if (i < 2 * D) {
                qs[i - D] = conv_channel(m, a, ring, g * D + (i - D), row, row0, pos, channels);
            } else if (i < 3 * D) {
                ks[i - 2 * D] = conv_channel(m, a, ring, (m.kv_head + g) * D + (i - 2 * D), row, row0, pos, channels);
            } else if (i < 3 * D + E) {
                const int x = i - 3 * D;
                vs[x] = conv_channel(m, a, ring, 2 * m.kv_head * D + h * E + x, row, row0, pos, channels);
            } else {
                const int x = i - 3 * D - E;
                const float z = m.g2 != nullptr ? low_rank(static_cast<const T*>(m.g2) + ((size_t)h * E + x) * m.gate_rank, pr + m.g_off, m.gate_rank)
                                                : pr[m.g_off + h * E + x];
                gate[x] = cm_gate(z, m.gate_act);
            }
        }
        const float beta = m.delta ? cm_sigmoid(pr[m.b_off + h]) : 1.0f;
        if (staged) cm_cp_wait_all();
        __syncthreads();
        if (write_ring && m.conv != nullptr) {         // a step of single tokens: this row's inputs enter the ring (nobody reads that entry in this step)
            float* entry = ring + (size_t)(pos % m.taps) * channels;
            if (h % share == 0)
                for (int i = threadIdx.x; i < 2 * D; i += blockDim.x) {
                    const int ch = i < D ? g * D + i : (m.kv_head + g) * D + (i - D);
                    entry[ch] = pr[ch];
                }
            for (int i = threadIdx.x; i < E; i += blockDim.x) entry[2 * m.kv_head * D + h * E + i] = pr[2 * m.kv_head * D + h * E + i];
        }
        float iq = m.q_scale, ik = 1.0f;
        if (m.unit) {                          // every warp sums for itself: no barrier
            float sq = 0.0f, sk = 0.0f;
            for (int d = lane; d < D; d += 32) {
                sq = fmaf(qs[d], qs[d], sq);
                sk = fmaf(ks[d], ks[d], sk);
            }
            iq = m.q_scale / sqrtf(lb_warp_sum(sq) + m.unit_eps);
            ik = 1.0f / sqrtf(lb_warp_sum(sk) + m.unit_eps);
        }
        float u = live ? vs[c] : 0.0f;
        if (m.delta) {
            float r = 0.0f;
            if (live)
                for (int d = ds; d < D; d += DS) r = fmaf(keep[d] * S[(size_t)d * E + c], ks[d], r);
            red[ds * ep2 + c] = r;
            __syncthreads();
            float sum = 0.0f;
            for (int i = 0; i < DS; ++i) sum += red[i * ep2 + c];
            u = beta * (u - ik * sum);
            __syncthreads();                   // red is used again below
        }
        u *= ik;
        float acc = 0.0f;
        if (live)
            for (int d = ds; d < D; d += DS) {
                const float s = fmaf(keep[d], S[(size_t)d * E + c], ks[d] * u);
                S[(size_t)d * E + c] = s;
                acc = fmaf(s, qs[d], acc);
            }
        red[ds * ep2 + c] = acc;
        __syncthreads();
        if (ds == 0 && live) {
            float sum = 0.0f;
            for (int i = 0; i < DS; ++i) sum += red[i * ep2 + c];
            os[c] = iq * sum;
        }
        __syncthreads();
        float ss = 0.0f;
        for (int x = lane; x < E; x += 32) ss = fmaf(os[x], os[x], ss);
        const float inv = 1.0f / sqrtf(lb_warp_sum(ss) / (float)E + m.eps);
        for (int x = threadIdx.x; x < E; x += blockDim.x) {
            const float o = os[x];
            if (a.o != nullptr) a.o[(size_t)row * a.ldo + h * E + x] = o;
            static_cast<T*>(a.heads)[(size_t)row * a.ldh + h * E + x] = lb_from_float<T>(o * inv * m.norm[x] * gate[x]);
        }
        __syncthreads();                       // the row's buffers are filled again
    }
    if (staged)
        for (int i = threadIdx.x; i < D * E; i += blockDim.x) st[i] = S[i];
}

// ---------------------------------------------------------------- the convolution's ring after a step with portions
__global__ void __launch_bounds__(256) channel_ring_kernel(lb_channel_memory m, StepArgs a) {
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const int seq = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x, channels = channels_of(m);
    const int row0 = a.q_start[seq], row1 = a.q_start[seq + 1];
    if (c >= channels) return;
    float* ring = a.state + (size_t)a.slots[seq] * m.slot_stride + (size_t)m.n_head * m.dim * m.vdim;
    for (int row = max(row0, row1 - m.taps); row < row1; ++row) ring[(size_t)(a.positions[row] % m.taps) * channels + c] = a.proj[(size_t)row * a.ld + c];
}

// ---------------------------------------------------------------- pieces of 32 rows
// Floats from the start of a (piece, head)'s scratch.  Under the delta rule U and the state lie in tiles of 16 value columns, as the scan's blocks read
// and write them: [tile][32][16] and [tile][dim][16]; without it [32][vdim] and [dim][vdim].
constexpr int kTileE = 16;
struct PieceLayout {
    int64_t p, q, keep, b, w, u, s, total;
};
__host__ __device__ inline PieceLayout piece_layout(int D, int E, int delta) {
    PieceLayout l{};
    int64_t at = 0;
    auto take = [&](int64_t n) { const int64_t r = at; at += (n + 3) / 4 * 4; return r; };
    const int64_t D4 = (D + 3) / 4 * 4, wide = delta ? (E + kTileE - 1) / kTileE * kTileE : E;
    l.p = take(kPiece * kPiece);                // P(t, j)
    l.q = take(kPiece * D);                     // exp(b_t) q_t
    l.keep = take(D);                           // exp(b_n)
    l.b = take(delta ? kPiece * D4 : 0);        // exp(b_n - b_j) k_j, rows of D4
    l.w = take(delta ? kPiece * D : 0);         // M K~, transposed: [dim][32]
    l.u = take(kPiece * wide);                  // V, or under the delta rule M V and after the scan U
    l.s = take(D * wide);                       // without the delta rule the piece's own sum; after the scan the state before the piece
    l.total = at;
    return l;
}

// Piece g of the step (pieces of 32 rows, request after request): its request and its number inside the request; false past the last.
__device__ __forceinline__ bool find_piece(const int32_t* q_start, int n_seq, int g, int* seq, int* piece) {
    for (int s = 0; s < n_seq; ++s) {
        const int pieces = (q_start[s + 1] - q_start[s] + kPiece - 1) / kPiece;
        if (g < pieces) {
            *seq = s;
            *piece = g;
            return true;
        }
        g -= pieces;
    }
    return false;
}

// acc[i][j] += a_i b_j over 4 x 4 results.
__device__ __forceinline__ void outer4(float (&acc)[4][4], const float4& a, const float4& b) {
    const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
}
// y[t][x] = sum_j m[t][j] v[j][x] for 4 rows from t0 and 4 columns (m [32][36] lower triangular, v at stride ldv, both on 16-byte borders).
__device__ __forceinline__ void tri_product(float (&y)[4][4], const float* m, const float* v, int ldv, int t0) {
    for (int j = 0; j < t0 + 4; j += 4) {
        float4 r[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) r[i] = *reinterpret_cast<const float4*>(m + (t0 + i) * 36 + j);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float4 b = *reinterpret_cast<const float4*>(v + (size_t)(j + k) * ldv);
            const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float rv = k == 0 ? r[i].x : k == 1 ? r[i].y : k == 2 ? r[i].z : r[i].w;
#pragma unroll
                for (int x = 0; x < 4; ++x) y[i][x] = fmaf(rv, bv[x], y[i][x]);
            }
        }
    }
}

// z[t][x] for eight rows t0 .. of column x: sum over a chunk of up to 32 of the rank; xT [32 r][36] holds the rows' inputs, w the column's weights.
__device__ __forceinline__ void rank_chunk(float (&z)[8], const float* xT, const float* w, int t0, int n) {
    for (int r = 0; r < n; ++r) {
        const float4 lo = *reinterpret_cast<const float4*>(xT + r * 36 + t0), hi = *reinterpret_cast<const float4*>(xT + r * 36 + t0 + 4);
        const float v = w[r];
        z[0] = fmaf(v, lo.x, z[0]); z[1] = fmaf(v, lo.y, z[1]); z[2] = fmaf(v, lo.z, z[2]); z[3] = fmaf(v, lo.w, z[3]);
        z[4] = fmaf(v, hi.x, z[4]); z[5] = fmaf(v, hi.y, z[5]); z[6] = fmaf(v, hi.z, z[6]); z[7] = fmaf(v, hi.w, z[7]);
    }
}
// A chunk of a low-rank map's operands: xT[r][t] = x[row0 + t][r0 + r] (zeros past the piece), w[c][r] = map[c][r0 + r] at stride 33.
template <typename T>
__device__ __forceinline__ void load_rank_chunk(float* xT, float* ws, const float* __restrict__ x, int64_t ldx, const T* __restrict__ map, int rank, int r0, int n_rows,
                                                int n_cols) {
    const int n = min(32, rank - r0);
    constexpr int B = 4;               // loads a thread has in flight before it stores the first
    for (int i0 = threadIdx.x; i0 < 32 * 32; i0 += B * blockDim.x) {
        float v[B];
#pragma unroll
        for (int k = 0; k < B; ++k) {
            const int i = i0 + k * blockDim.x, t = i >> 5, r = i & 31;
            v[k] = i < 32 * 32 && t < n_rows && r < n ? x[(size_t)t * ldx + r0 + r] : 0.0f;
        }
#pragma unroll
        for (int k = 0; k < B; ++k) {
            const int i = i0 + k * blockDim.x;
            if (i < 32 * 32) xT[(i & 31) * 36 + (i >> 5)] = v[k];
        }
    }
    for (int i0 = threadIdx.x; i0 < n_cols * 32; i0 += 2 * B * blockDim.x) {
        T v[2 * B];
#pragma unroll
        for (int k = 0; k < 2 * B; ++k) {
            const int i = i0 + k * blockDim.x, c = i >> 5, r = i & 31;
            v[k] = i < n_cols * 32 && r < n ? map[(size_t)c * rank + r0 + r] : lb_from_float<T>(0.0f);
        }
#pragma unroll
        for (int k = 0; k < 2 * B; ++k) {
            const int i = i0 + k * blockDim.x;
            if (i < n_cols * 32) ws[(i >> 5) * 33 + (i & 31)] = lb_to_float(v[k]);
        }
    }
}

__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// A piece's own matrices, from the projection's rows on: convolution, unit vectors and decays, the pairs' products, the triangle's solution.
template <typename T, bool DELTA>
__global__ void __launch_bounds__(256) channel_pieces_kernel(lb_channel_memory m, StepArgs a, float* __restrict__ scratch, int n_seq) {
    extern __shared__ __align__(16) float smem[];
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    int seq, piece;
    if (!find_piece(a.q_start, n_seq, blockIdx.x, &seq, &piece)) return;
    const int h = blockIdx.y, D = m.dim, E = m.vdim, D4 = (D + 3) / 4 * 4, E4 = (E + 3) / 4 * 4, LD = D4 + 4, LE = E4 + 4, g = h / (m.n_head / m.kv_head), channels = channels_of(m);
    const int first = a.q_start[seq], row0 = first + piece * kPiece, n = min(kPiece, a.q_start[seq + 1] - row0), pos0 = a.positions[row0];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* Am = smem;                          // [32][36]; before the pairs the decays' inputs [32 r][36]
    float* M = Am + kPiece * 36;               // [32][36]
    float* beta = M + kPiece * 36;             // [32]
    float* qs = beta + kPiece;                 // [32][LD]
    float* ks = qs + kPiece * LD;              // [32][LD]
    float* bs = ks + kPiece * LD;              // [32][LD] log decays, then their running sums
    float* vs = bs + kPiece * LD;              // [32][LE]
    float* fs = vs + kPiece * LE;              // [48][LD] rows with one half of a pair's exponential; before that the decays' map [D][33]
    // Rows start on 16-byte borders, columns up to the next multiple of four are zeros.
    if (D4 > D || E4 > E) {
        for (int t = warp; t < kPiece; t += 8) {
            if (lane < D4 - D) qs[t * LD + D + lane] = ks[t * LD + D + lane] = bs[t * LD + D + lane] = 0.0f;
            if (lane < E4 - E) vs[t * LE + E + lane] = 0.0f;
        }
    }
    const PieceLayout l = piece_layout(D, E, DELTA);
    float* out = scratch + ((size_t)blockIdx.x * m.n_head + h) * l.total;
    const float* slot = a.state + (size_t)a.slots[seq] * m.slot_stride;
    const float* ring = slot + (size_t)m.n_head * D * E;
    // Queries, keys and values: eight rows of a channel an item, the convolution's earlier inputs in registers.
    for (int i = threadIdx.x; i < 4 * (2 * D + E); i += blockDim.x) {
        const int part = i / (2 * D + E), x = i - part * (2 * D + E), t0 = 8 * part;
        const int c = x < D ? g * D + x : x < 2 * D ? (m.kv_head + g) * D + (x - D) : 2 * m.kv_head * D + h * E + (x - 2 * D);
        float* dst = x < D ? qs + x : x < 2 * D ? ks + (x - D) : vs + (x - 2 * D);
        const int ld = x < 2 * D ? LD : LE;
        const float* col = a.proj + (size_t)row0 * a.ld + c;
        auto input = [&](int t) -> float {     // the channel's input at row row0 + t: of this step, of an earlier one, or before the start
            if (row0 + t >= first) return t < n ? col[(int64_t)t * a.ld] : 0.0f;
            const int p = pos0 + t;
            return p >= 0 ? ring[(size_t)(p % m.taps) * channels + c] : 0.0f;
        };
        if (m.conv == nullptr) {
            float u[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) u[k] = input(t0 + k);
#pragma unroll
            for (int k = 0; k < 8; ++k) dst[(t0 + k) * ld] = u[k];
        } else if (m.taps <= 4) {
            float u[11], w[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) w[k] = k < m.taps ? m.conv[(size_t)c * m.taps + m.taps - 1 - k] : 0.0f;      // w[k]: of the input k tokens ago
#pragma unroll
            for (int k = 0; k < 11; ++k) u[k] = k >= 4 - m.taps ? input(t0 + k - 3) : 0.0f;
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                const float z = fmaf(w[3], u[k], fmaf(w[2], u[k + 1], fmaf(w[1], u[k + 2], w[0] * u[k + 3])));
                dst[(t0 + k) * ld] = t0 + k < n ? z * cm_sigmoid(z) : 0.0f;
            }
        } else {
            for (int k = 0; k < 8; ++k) {
                float z = 0.0f;
                for (int j = 0; j < m.taps; ++j) z = fmaf(m.conv[(size_t)c * m.taps + j], input(t0 + k - (m.taps - 1) + j), z);
                dst[(t0 + k) * ld] = t0 + k < n ? z * cm_sigmoid(z) : 0.0f;
            }
        }
    }
    if (DELTA && threadIdx.x < kPiece) beta[threadIdx.x] = threadIdx.x < n ? cm_sigmoid(a.proj[(size_t)(row0 + threadIdx.x) * a.ld + m.b_off + h]) : 0.0f;
    // The decays: the low-rank map in chunks of 32 of its rank, eight rows of a channel an item.
    const float a_exp = m.a_log != nullptr ? expf(m.a_log[h]) * kLbLog2e : kLbLog2e / m.tau;
    for (int r0 = 0; r0 < m.rank; r0 += 32) {
        if (r0 > 0) __syncthreads();
        load_rank_chunk(Am, fs, a.proj + (size_t)row0 * a.ld + m.a_off, a.ld, static_cast<const T*>(m.a2) + (size_t)h * D * m.rank, m.rank, r0, n, D);
        __syncthreads();
        for (int i = threadIdx.x; i < 4 * D; i += blockDim.x) {
            const int part = i / D, d = i - part * D, t0 = 8 * part;
            float z[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) z[k] = r0 > 0 ? bs[(t0 + k) * LD + d] : m.z_bias != nullptr ? m.z_bias[h * D + d] : 0.0f;
            rank_chunk(z, Am, fs + d * 33, t0, min(32, m.rank - r0));
            if (r0 + 32 >= m.rank) {
#pragma unroll
                for (int k = 0; k < 8; ++k) z[k] = t0 + k < n ? -a_exp * (m.a_log != nullptr ? lb_softplus(z[k]) : lb_softplus(-z[k])) : 0.0f;
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) bs[(t0 + k) * LD + d] = z[k];
        }
    }
    __syncthreads();
    if (m.unit) {
        for (int t = warp; t < n; t += 8) {
            float sq = 0.0f, sk = 0.0f;
            for (int d = lane; d < D; d += 32) {
                sq = fmaf(qs[t * LD + d], qs[t * LD + d], sq);
                sk = fmaf(ks[t * LD + d], ks[t * LD + d], sk);
            }
            const float iq = 1.0f / sqrtf(lb_warp_sum(sq) + m.unit_eps), ik = 1.0f / sqrtf(lb_warp_sum(sk) + m.unit_eps);
            for (int d = lane; d < D; d += 32) {
                qs[t * LD + d] *= iq;
                ks[t * LD + d] *= ik;
            }
        }
    }
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        float b = 0.0f;
#pragma unroll
        for (int t = 0; t < kPiece; ++t) {
            b += bs[t * LD + d];
            bs[t * LD + d] = b;
        }
    }
    __syncthreads();
    // The pairs.  Rows of the second half meet keys of the first through the border between them: exp(b_t - b_j) = exp(b_t - b_15) exp(b_15 - b_j), both
    // exponents at most 0, so those 256 pairs are plain products; pairs inside a half make their exponentials one by one.
    constexpr int kHalf = kPiece / 2;
    for (int t = warp; t < kHalf; t += 8)
        for (int d = lane; d < D4; d += 32) {
            const float border = bs[(kHalf - 1) * LD + d], e = fast_exp2(bs[(kHalf + t) * LD + d] - border);
            fs[t * LD + d] = qs[(kHalf + t) * LD + d] * e;
            if (DELTA) fs[(kHalf + t) * LD + d] = ks[(kHalf + t) * LD + d] * e;
            fs[(2 * kHalf + t) * LD + d] = ks[t * LD + d] * fast_exp2(border - bs[t * LD + d]);
        }
    __syncthreads();
    auto dot4 = [](const float4& x, const float4& y, float sum) { return fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, sum)))); };
    {
        const int t = threadIdx.x >> 4, j = threadIdx.x & 15;
        const float4 *qt = reinterpret_cast<const float4*>(fs + t * LD), *kt = reinterpret_cast<const float4*>(fs + (kHalf + t) * LD);
        const float4* kj = reinterpret_cast<const float4*>(fs + (2 * kHalf + j) * LD);
        float p = 0.0f, av = 0.0f;
#pragma unroll 4
        for (int d = 0; d < D4 / 4; ++d) {
            const float4 k = kj[d];
            p = dot4(qt[d], k, p);
            if (DELTA) av = dot4(kt[d], k, av);
        }
        out[l.p + (kHalf + t) * kPiece + j] = p * m.q_scale;
        out[l.p + t * kPiece + kHalf + j] = 0.0f;
        if (DELTA) {
            Am[(kHalf + t) * 36 + j] = av;
            Am[t * 36 + kHalf + j] = 0.0f;
        }
    }
    for (int r = warp; r < kHalf; r += 8) {    // a warp: row r of the first half and row r of the second, a half of the lanes each
        const int half = lane >> 4 << 4, t = half + r, j = half + (lane & 15);
        float p = 0.0f, av = 0.0f;
        if (j <= t && t < n) {
            const float4 *qt = reinterpret_cast<const float4*>(qs + t * LD), *kt = reinterpret_cast<const float4*>(ks + t * LD);
            const float4 *bt = reinterpret_cast<const float4*>(bs + t * LD), *kj = reinterpret_cast<const float4*>(ks + j * LD);
            const float4* bj = reinterpret_cast<const float4*>(bs + j * LD);
#pragma unroll 2
            for (int d = 0; d < D4 / 4; ++d) {
                const float4 x = bt[d], y = bj[d], k = kj[d];
                const float4 e = make_float4(fast_exp2(x.x - y.x) * k.x, fast_exp2(x.y - y.y) * k.y, fast_exp2(x.z - y.z) * k.z, fast_exp2(x.w - y.w) * k.w);
                p = dot4(qt[d], e, p);
                if (DELTA) av = dot4(kt[d], e, av);
            }
        }
        out[l.p + t * kPiece + j] = p * m.q_scale;
        if (DELTA) Am[t * 36 + j] = j < t ? av : 0.0f;
    }
    __syncthreads();
    // Warp 0 solves the triangle, a column a lane; the others turn the rows into what the scan and the outputs read.
    if (DELTA && warp == 0) {
        float x[kPiece];
#pragma unroll
        for (int t = 0; t < kPiece; ++t) {
            float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
            for (int j = 0; j < t; ++j) {
                if (j & 1) s1 = fmaf(Am[t * 36 + j], x[j], s1);
                else s0 = fmaf(Am[t * 36 + j], x[j], s0);
            }
            x[t] = beta[t] * ((t == lane ? 1.0f : 0.0f) - (s0 + s1));
            M[t * 36 + lane] = x[t];
        }
    } else {
        for (int t = DELTA ? warp - 1 : warp; t < kPiece; t += DELTA ? 7 : 8)
            for (int d = lane; d < (DELTA ? D4 : D); d += 32) {
                const float b = bs[t * LD + d], b_last = bs[(kPiece - 1) * LD + d], k = ks[t * LD + d], e = fast_exp2(b), kb = fast_exp2(b_last - b) * k;
                if (d < D) out[l.q + t * D + d] = qs[t * LD + d] * m.q_scale * e;
                if (DELTA) {
                    out[l.b + t * D4 + d] = kb;
                    ks[t * LD + d] = k * e;        // K~
                } else {
                    ks[t * LD + d] = kb;
                }
                if (t == 0 && d < D) out[l.keep + d] = fast_exp2(b_last);
            }
    }
    __syncthreads();
    if (DELTA) {
        // M K~ and M V: thread (four rows, four columns).
        const int tiles_d = D4 / 4, tiles = tiles_d + E4 / 4;
        for (int i = threadIdx.x; i < 8 * tiles; i += blockDim.x) {
            const int part = i / tiles, x = i - part * tiles, t0 = 4 * part;
            float y[4][4] = {};
            if (x < tiles_d) tri_product(y, M, ks + 4 * x, LD, t0);
            else tri_product(y, M, vs + 4 * (x - tiles_d), LE, t0);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                if (x < tiles_d) {
                    if (4 * x + k < D) *reinterpret_cast<float4*>(out + l.w + (4 * x + k) * kPiece + t0) = make_float4(y[0][k], y[1][k], y[2][k], y[3][k]);
                } else {
                    const int c = 4 * (x - tiles_d);
                    *reinterpret_cast<float4*>(out + l.u + (c / kTileE * kPiece + t0 + k) * kTileE + c % kTileE) = make_float4(y[k][0], y[k][1], y[k][2], y[k][3]);
                }
            }
        }
    } else {
        for (int t = warp; t < kPiece; t += 8)
            for (int x = lane; x < E; x += 32) out[l.u + t * E + x] = vs[t * LE + x];
        // The piece's own sum: thread (four channels, four columns).
        const int tiles_e = E4 / 4;
        for (int i = threadIdx.x; i < D4 / 4 * tiles_e; i += blockDim.x) {
            const int part = i / tiles_e, x = 4 * (i - part * tiles_e), d0 = 4 * part;
            float y[4][4] = {};
#pragma unroll 4
            for (int j = 0; j < n; ++j) outer4(y, *reinterpret_cast<const float4*>(ks + j * LD + d0), *reinterpret_cast<const float4*>(vs + j * LE + x));
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
                for (int v = 0; v < 4; ++v)
                    if (d0 + k < D && x + v < E) out[l.s + (d0 + k) * E + x + v] = y[k][v];
        }
    }
}

// The scan without the delta rule: every element of S by itself, S <- exp(b_n)[d] S + sum, the state before every piece left in the sum's place.
constexpr int kAhead = 8;
__global__ void __launch_bounds__(256) channel_scan_kernel(lb_channel_memory m, StepArgs a, float* __restrict__ scratch) {
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const int seq = blockIdx.x, h = blockIdx.y, D = m.dim, E = m.vdim, i = blockIdx.z * blockDim.x + threadIdx.x;
    const int pieces = (a.q_start[seq + 1] - a.q_start[seq] + kPiece - 1) / kPiece;
    if (pieces <= 0 || i >= D * E) return;
    int g0 = 0;
    for (int s = 0; s < seq; ++s) g0 += (a.q_start[s + 1] - a.q_start[s] + kPiece - 1) / kPiece;
    const PieceLayout l = piece_layout(D, E, 0);
    float* st = a.state + (size_t)a.slots[seq] * m.slot_stride + (size_t)h * D * E + i;
    const size_t stride = (size_t)m.n_head * l.total;
    float* first = scratch + ((size_t)g0 * m.n_head + h) * l.total;
    const int d = i / E;
    float S = *st;
    for (int p0 = 0; p0 < pieces; p0 += kAhead) {
        float sum[kAhead], keep[kAhead];
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            const float* at = first + (size_t)min(p0 + k, pieces - 1) * stride;
            sum[k] = at[l.s + i];
            keep[k] = at[l.keep + d];
        }
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            if (p0 + k >= pieces) break;
            first[(size_t)(p0 + k) * stride + l.s + i] = S;
            S = fmaf(keep[k], S, sum[k]);
        }
    }
    *st = S;
}

// The scan under the delta rule: a block per (request, head, tile of 16 value columns) walks the request's pieces, U = M V - (M K~) S, then
// S <- exp(b_n) S + sum_j (exp(b_n - b_j) k_j) u_j^T; the next piece's matrices travel while this one is added.  Both products are made in 4 x 4 results a
// thread (a 16-byte read of shared memory costs as much as four plain ones), the reduction cut over warps (over groups of threads for S) whose shares
// meet in shared memory in a fixed order.
__global__ void __launch_bounds__(256) delta_scan_kernel(lb_channel_memory m, StepArgs a, float* __restrict__ scratch) {
    extern __shared__ __align__(16) float smem[];
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    constexpr int VT = kTileE;
    const int seq = blockIdx.x, h = blockIdx.y, D = m.dim, E = m.vdim, c0 = blockIdx.z * VT;
    const int pieces = (a.q_start[seq + 1] - a.q_start[seq] + kPiece - 1) / kPiece;
    if (pieces <= 0) return;
    int g0 = 0;
    for (int s = 0; s < seq; ++s) g0 += (a.q_start[s + 1] - a.q_start[s] + kPiece - 1) / kPiece;
    const PieceLayout l = piece_layout(D, E, 1);
    const int D4 = (D + 3) / 4 * 4, matrices = D4 + kPiece * (D4 + D);        // keep, B and W lie one after the other
    float* S = smem;                           // [D4][VT]
    float* U = S + D4 * VT;                    // [32][VT]
    float* red = U + kPiece * VT;              // [8][32][VT], or [groups][D4][VT]
    float* buf = red + 8 * kPiece * VT;        // [2][keep | B | W^T | M V's columns]
    const int buf_floats = matrices + kPiece * VT;
    const size_t stride = (size_t)m.n_head * l.total, u_tile = l.u + (size_t)blockIdx.z * kPiece * VT, s_tile = l.s + (size_t)blockIdx.z * D * VT;
    float* first = scratch + ((size_t)g0 * m.n_head + h) * l.total;
    float* st = a.state + (size_t)a.slots[seq] * m.slot_stride + (size_t)h * D * E;
    auto ask = [&](int p) {
        const float* src = first + (size_t)p * stride;
        float* dst = buf + (p & 1) * buf_floats;
        for (int i = threadIdx.x; i < matrices / 4; i += 256) cm_cp_async16(dst + 4 * i, src + l.keep + 4 * i);
        if (threadIdx.x < kPiece * VT / 4) cm_cp_async16(dst + matrices + 4 * threadIdx.x, src + u_tile + 4 * threadIdx.x);
        cm_cp_commit();
    };
    ask(0);
    for (int i = threadIdx.x; i < D4 * VT; i += blockDim.x) {
        const int d = i / VT, x = i - d * VT;
        S[i] = d < D && c0 + x < E ? st[(size_t)d * E + c0 + x] : 0.0f;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lt = 4 * (lane >> 2), lc = 4 * (lane & 3);
    // S: tile (4 channels, 4 columns) of the thread, and its share of the rows.
    const int tiles = D4, tile = threadIdx.x % tiles, group = threadIdx.x / tiles, d0 = 4 * (tile >> 2), x0 = 4 * (tile & 3);
    int groups = 1;
    while (2 * groups * tiles <= 256 && groups < 8) groups *= 2;
    const int share = kPiece / groups;
    for (int p = 0; p < pieces; ++p) {
        cm_cp_wait_all();
        __syncthreads();                       // the piece has arrived; S is whole; the other buffer is free
        if (p + 1 < pieces) ask(p + 1);
        const float* keep = buf + (p & 1) * buf_floats;
        const float* B = keep + D4;            // [32][D4]
        const float* W = B + kPiece * D4;      // [D][32]
        const float* MV = keep + matrices;
        float* at = first + (size_t)p * stride;
        for (int i = threadIdx.x; i < D * VT / 4; i += 256) *reinterpret_cast<float4*>(at + s_tile + 4 * i) = *reinterpret_cast<const float4*>(S + 4 * i);
        float y[4][4] = {};
#pragma unroll 4
        for (int d = warp; d < D; d += 8) outer4(y, *reinterpret_cast<const float4*>(W + d * kPiece + lt), *reinterpret_cast<const float4*>(S + d * VT + lc));
#pragma unroll
        for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(red + (warp * kPiece + lt + i) * VT + lc) = make_float4(y[i][0], y[i][1], y[i][2], y[i][3]);
        __syncthreads();
        if (threadIdx.x < kPiece * VT / 4) {
            float4 u = *reinterpret_cast<const float4*>(MV + 4 * threadIdx.x);
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float4 r = *reinterpret_cast<const float4*>(red + w * kPiece * VT + 4 * threadIdx.x);
                u.x -= r.x; u.y -= r.y; u.z -= r.z; u.w -= r.w;
            }
            *reinterpret_cast<float4*>(U + 4 * threadIdx.x) = u;
            *reinterpret_cast<float4*>(at + u_tile + 4 * threadIdx.x) = u;
        }
        __syncthreads();
        float z[4][4] = {};
        if (group < groups) {
#pragma unroll 8
            for (int t = group * share; t < (group + 1) * share; ++t)
                outer4(z, *reinterpret_cast<const float4*>(B + t * D4 + d0), *reinterpret_cast<const float4*>(U + t * VT + x0));
        }
        if (groups > 1) {
            if (group < groups) {
#pragma unroll
                for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(red + (group * D4 + d0 + i) * VT + x0) = make_float4(z[i][0], z[i][1], z[i][2], z[i][3]);
            }
            __syncthreads();
            for (int i = threadIdx.x; i < D4 * VT / 4; i += 256) {
                const float k = keep[i >> 2];
                float4 v = *reinterpret_cast<const float4*>(red + 4 * i), old = *reinterpret_cast<const float4*>(S + 4 * i);
                for (int g = 1; g < groups; ++g) {
                    const float4 r = *reinterpret_cast<const float4*>(red + g * D4 * VT + 4 * i);
                    v.x += r.x; v.y += r.y; v.z += r.z; v.w += r.w;
                }
                *reinterpret_cast<float4*>(S + 4 * i) = make_float4(fmaf(k, old.x, v.x), fmaf(k, old.y, v.y), fmaf(k, old.z, v.z), fmaf(k, old.w, v.w));
            }
        } else {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float k = keep[d0 + i];
                float4* dst = reinterpret_cast<float4*>(S + (d0 + i) * VT + x0);
                *dst = make_float4(fmaf(k, dst->x, z[i][0]), fmaf(k, dst->y, z[i][1]), fmaf(k, dst->z, z[i][2]), fmaf(k, dst->w, z[i][3]));
            }
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < D * VT; i += blockDim.x) {
        const int d = i / VT, x = i - d * VT;
        if (c0 + x < E) st[(size_t)d * E + c0 + x] = S[i];
    }
}

// The outputs of a piece with the heads' norm and gate.  Thread (c, tg) owns column c for the R rows tg R .. tg R + R - 1; the state before the piece
// and U come to shared memory (`staged`) while the gates are made.
template <typename T, int R>
__global__ void __launch_bounds__(256) channel_outputs_kernel(lb_channel_memory m, StepArgs a, float* __restrict__ scratch, int n_seq, int staged) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float inv[kPiece];
    constexpr int EP = 8 * R;                  // threads across the columns: 256 / (32 / R)
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    int seq, piece;
    if (!find_piece(a.q_start, n_seq, blockIdx.x, &seq, &piece)) return;
    const int h = blockIdx.y, D = m.dim, E = m.vdim, d4 = (D + 3) / 4 * 4;
    const int row0 = a.q_start[seq] + piece * kPiece, n = min(kPiece, a.q_start[seq + 1] - row0);
    float* P = smem;                           // [32][32]
    float* qs = P + kPiece * kPiece;           // [32][d4]
    float* xT = qs + kPiece * d4;              // [32][36] the gates' inputs
    float* gw = xT + 32 * 36;                  // [E][33] their map
    float* os = gw;                            // [32][E + 1] afterwards
    float* Ss = gw + ((E > 32 ? E : 32) * 33 + 35) / 4 * 4;      // [D][E]
    const PieceLayout l = piece_layout(D, E, m.delta);
    const float* in = scratch + ((size_t)blockIdx.x * m.n_head + h) * l.total;
    cm_fetch(P, in + l.p, kPiece * kPiece);
    if (D == d4) {
        cm_fetch(qs, in + l.q, kPiece * D);
    } else {
        for (int i = threadIdx.x; i < kPiece * d4; i += blockDim.x) {
            const int t = i / d4, d = i - t * d4;
            if (d < D) cm_cp_async4(qs + i, in + l.q + t * D + d);
            else qs[i] = 0.0f;
        }
    }
    const int wide = m.delta ? (E + kTileE - 1) / kTileE * kTileE : E;
    float* Us = Ss + (D * wide + 3) / 4 * 4;   // [32][E], or in tiles
    if (staged) {
        cm_fetch(Ss, in + l.s, D * wide);
        cm_fetch(Us, in + l.u, kPiece * wide);
    }
    cm_cp_commit();
    const int c = threadIdx.x % EP, t0 = threadIdx.x / EP * R;
    float gate[R];
#pragma unroll
    for (int i = 0; i < R; ++i) gate[i] = 0.0f;
    if (m.g2 != nullptr) {
        for (int r0 = 0; r0 < m.gate_rank; r0 += 32) {
            if (r0 > 0) __syncthreads();
            load_rank_chunk(xT, gw, a.proj + (size_t)row0 * a.ld + m.g_off, a.ld, static_cast<const T*>(m.g2) + (size_t)h * E * m.gate_rank, m.gate_rank, r0, n, E);
            __syncthreads();
            if (c < E) {
                const int count = min(32, m.gate_rank - r0);
                for (int r = 0; r < count; ++r) {
                    const float w = gw[c * 33 + r];
                    if constexpr (R % 4 == 0) {
#pragma unroll
                        for (int i = 0; i < R; i += 4) {
                            const float4 x = *reinterpret_cast<const float4*>(xT + r * 36 + t0 + i);
                            gate[i] = fmaf(w, x.x, gate[i]);
                            gate[i + 1] = fmaf(w, x.y, gate[i + 1]);
                            gate[i + 2] = fmaf(w, x.z, gate[i + 2]);
                            gate[i + 3] = fmaf(w, x.w, gate[i + 3]);
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < R; ++i) gate[i] = fmaf(w, xT[r * 36 + t0 + i], gate[i]);
                    }
                }
            }
        }
    } else if (c < E) {
#pragma unroll
        for (int i = 0; i < R; ++i) gate[i] = t0 + i < n ? a.proj[(size_t)(row0 + t0 + i) * a.ld + m.g_off + h * E + c] : 0.0f;
    }
    cm_cp_wait_all();
    __syncthreads();
    float y[R];
#pragma unroll
    for (int i = 0; i < R; ++i) y[i] = 0.0f;
    if (c < E) {
        // Column c of the state and of U: in its tile under the delta rule.
        const int ld = m.delta ? kTileE : E;
        const float* S = (staged ? Ss : in + l.s) + (m.delta ? c / kTileE * D * kTileE + c % kTileE : c);
#pragma unroll 2
        for (int d = 0; d < D; d += 4) {
            float s[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) s[k] = d + k < D ? S[(d + k) * ld] : 0.0f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const float4 q = *reinterpret_cast<const float4*>(qs + (t0 + i) * d4 + d);
                y[i] = fmaf(q.x, s[0], fmaf(q.y, s[1], fmaf(q.z, s[2], fmaf(q.w, s[3], y[i]))));
            }
        }
        const float* u = (staged ? Us : in + l.u) + (m.delta ? c / kTileE * kPiece * kTileE + c % kTileE : c);
        const int last = min(n, t0 + R);       // rows after the last of this thread's are not seen
#pragma unroll 2
        for (int j = 0; j < last; j += 4) {
            float s[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) s[k] = j + k < n ? u[(j + k) * ld] : 0.0f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const float4 p = *reinterpret_cast<const float4*>(P + (t0 + i) * kPiece + j);
                y[i] = fmaf(p.x, s[0], fmaf(p.y, s[1], fmaf(p.z, s[2], fmaf(p.w, s[3], y[i]))));
            }
        }
#pragma unroll
        for (int i = 0; i < R; ++i) os[(t0 + i) * (E + 1) + c] = y[i];
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t = warp; t < n; t += 8) {
        const float* o = os + t * (E + 1);
        float ss = 0.0f;
        for (int x = lane; x < E; x += 32) ss = fmaf(o[x], o[x], ss);
        ss = lb_warp_sum(ss);
        if (lane == 0) inv[t] = 1.0f / sqrtf(ss / (float)E + m.eps);
    }
    __syncthreads();
    if (c >= E) return;
    const float gain = m.norm[c];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        if (t0 + i >= n) break;
        const size_t row = (size_t)(row0 + t0 + i);
        if (a.o != nullptr) a.o[row * a.ldo + h * E + c] = y[i];
        static_cast<T*>(a.heads)[row * a.ldh + h * E + c] = lb_from_float<T>(y[i] * inv[t0 + i] * gain * cm_gate(gate[i], m.gate_act));
    }
}

int check_shape(const lb_channel_memory* m) {
    LB_CHECK_ARG(m != nullptr && m->n_head > 0 && m->kv_head > 0 && m->n_head % m->kv_head == 0 && m->dim > 0 && m->dim <= 256 && m->vdim > 0 && m->vdim <= 256,
                 "channel memory: heads of up to 256 values, query and key heads that divide the heads");
    LB_CHECK_ARG(m->a2 != nullptr && m->rank > 0 && m->norm != nullptr && (m->g2 == nullptr || m->gate_rank > 0) && (m->a_log != nullptr || m->tau > 0.0f),
                 "channel memory: the decays' map, the heads' gain or a constant is missing");
    LB_CHECK_ARG(m->conv == nullptr || m->taps >= 1, "channel memory: %d taps", m->taps);
    LB_CHECK_ARG(m->gate_act == LB_GATE_SIGMOID || m->gate_act == LB_GATE_SILU, "channel memory: gate %d (0 sigmoid, 1 silu)", m->gate_act);
    const int64_t need = (int64_t)m->n_head * m->dim * m->vdim + (m->conv != nullptr ? (int64_t)m->taps * (2 * m->kv_head * m->dim + m->n_head * m->vdim) : 0);
    LB_CHECK_ARG(m->slot_stride >= need, "channel memory: the state slots are too small");
    return LB_OK;
}

StepArgs step_of(const lb_channel_step* s) {
    return StepArgs{s->proj, s->ld, s->positions, s->tok_seq, s->q_start, s->slots, s->state, s->o, s->ldo, s->heads, s->ldh};
}

int launch_ring(const lb_channel_memory& m, const StepArgs& a, int n_seq, cudaStream_t s) {
    const int channels = 2 * m.kv_head * m.dim + m.n_head * m.vdim;
    LB_CHECK_CUDA(lb_launch_overlapped(channel_ring_kernel, dim3(n_seq, (channels + 255) / 256), dim3(256), 0, s, m, a));
    return LB_OK;
}

}  // namespace

extern "C" int lb_channel_memory_rows(int dtype, const lb_channel_memory* memory, const lb_channel_step* step, int n_seq, int decode_only, void* stream) {
    if (int rc = check_shape(memory)) return rc;
    LB_CHECK_ARG(dtype == LB_F32 || dtype == LB_BF16, "channel memory: unknown dtype %d", dtype);
    if (n_seq == 0) return LB_OK;
    const lb_channel_memory m = *memory;
    const StepArgs a = step_of(step);
    auto s = static_cast<cudaStream_t>(stream);
    int ep2 = 1;
    while (ep2 < m.vdim) ep2 <<= 1;
    const int threads = 3 * m.dim + 2 * m.vdim > 256 ? 512 : 256;      // a thread a value of the row's queries, keys, decays, values and gates
    const size_t base = (3 * ((size_t)m.dim + m.vdim) + threads + 3) / 4 * 4 * sizeof(float), with_state = base + (size_t)m.dim * m.vdim * sizeof(float);
    const int staged = with_state <= 160 * 1024 ? 1 : 0;
    const size_t smem = staged ? with_state : base;
    auto launch = [&](auto kernel) -> int {
        if (smem > 48 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, dim3(n_seq, m.n_head), dim3(threads), smem, s, m, a, ep2, staged, decode_only));
        return LB_OK;
    };
    if (int rc = dtype == LB_F32 ? launch(channel_memory_rows_kernel<float>) : launch(channel_memory_rows_kernel<__nv_bfloat16>)) return rc;
    if (m.conv != nullptr && !decode_only) return launch_ring(m, a, n_seq, s);
    return LB_OK;
}

extern "C" int64_t lb_channel_memory_pieces_floats(int n_tokens, int n_seq, int n_head, int dim, int vdim, int delta) {
    return ((int64_t)n_tokens / kPiece + n_seq) * n_head * piece_layout(dim, vdim, delta).total;
}

extern "C" int lb_channel_memory_pieces(int dtype, const lb_channel_memory* memory, const lb_channel_step* step, float* scratch, int n_tokens, int n_seq,
                                        void* stream) {
    if (int rc = check_shape(memory)) return rc;
    LB_CHECK_ARG(dtype == LB_F32 || dtype == LB_BF16, "channel memory: unknown dtype %d", dtype);
    LB_CHECK_ARG(scratch != nullptr, "channel memory in pieces: scratch is missing");
    if (n_seq == 0 || n_tokens == 0) return LB_OK;
    const lb_channel_memory m = *memory;
    const StepArgs a = step_of(step);
    auto s = static_cast<cudaStream_t>(stream);
    const int pieces = n_tokens / kPiece + n_seq, D = m.dim, E = m.vdim, d4 = (D + 3) / 4 * 4;
    auto launch = [&](auto kernel, dim3 grid, size_t smem, auto... args) -> int {
        LB_CHECK_ARG(smem <= 220 * 1024, "channel memory in pieces: heads of %d x %d values do not fit shared memory", D, E);
        if (smem > 48 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, grid, dim3(256), smem, s, args...));
        return LB_OK;
    };
    const dim3 grid(pieces, m.n_head);
    const size_t own = (2 * kPiece * 36 + kPiece + (3 * (size_t)kPiece + 48) * (d4 + 4) + (size_t)kPiece * ((E + 3) / 4 * 4 + 4)) * sizeof(float);
    if (m.delta) {
        if (int rc = dtype == LB_F32 ? launch(channel_pieces_kernel<float, true>, grid, own, m, a, scratch, n_seq)
                                     : launch(channel_pieces_kernel<__nv_bfloat16, true>, grid, own, m, a, scratch, n_seq)) return rc;
        const size_t scan = ((size_t)d4 * kTileE + 9 * (size_t)kPiece * kTileE + 2 * (d4 + (size_t)kPiece * (d4 + D) + kPiece * kTileE)) * sizeof(float);
        if (int rc = launch(delta_scan_kernel, dim3(n_seq, m.n_head, (E + kTileE - 1) / kTileE), scan, m, a, scratch)) return rc;
    } else {
        if (int rc = dtype == LB_F32 ? launch(channel_pieces_kernel<float, false>, grid, own, m, a, scratch, n_seq)
                                     : launch(channel_pieces_kernel<__nv_bfloat16, false>, grid, own, m, a, scratch, n_seq)) return rc;
        if (int rc = launch(channel_scan_kernel, dim3(n_seq, m.n_head, (D * E + 255) / 256), 0, m, a, scratch)) return rc;
    }
    // The ring only after the pieces have read it.
    if (m.conv != nullptr)
        if (int rc = launch_ring(m, a, n_seq, s)) return rc;
    const size_t base = (kPiece * kPiece + (size_t)kPiece * d4 + 32 * 36 + ((E > 32 ? E : 32) * 33 + 35) / 4 * 4) * sizeof(float);
    const int wide = m.delta ? (E + kTileE - 1) / kTileE * kTileE : E;
    const size_t with_state = base + ((size_t)(D * wide + 3) / 4 * 4 + (size_t)kPiece * wide) * sizeof(float);
    const int staged = with_state <= 110 * 1024 ? 1 : 0;
    const size_t outs = staged ? with_state : base;
#define LB_OUTPUTS(T)                                                                                 \
    (E <= 8     ? launch(channel_outputs_kernel<T, 1>, grid, outs, m, a, scratch, n_seq, staged)      \
     : E <= 16  ? launch(channel_outputs_kernel<T, 2>, grid, outs, m, a, scratch, n_seq, staged)      \
     : E <= 32  ? launch(channel_outputs_kernel<T, 4>, grid, outs, m, a, scratch, n_seq, staged)      \
     : E <= 64  ? launch(channel_outputs_kernel<T, 8>, grid, outs, m, a, scratch, n_seq, staged)      \
     : E <= 128 ? launch(channel_outputs_kernel<T, 16>, grid, outs, m, a, scratch, n_seq, staged)     \
                : launch(channel_outputs_kernel<T, 32>, grid, outs, m, a, scratch, n_seq, staged))
    return dtype == LB_F32 ? LB_OUTPUTS(float) : LB_OUTPUTS(__nv_bfloat16);
#undef LB_OUTPUTS
}
