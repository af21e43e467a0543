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
// Launches: the low-rank maps, the convolution, the pieces' own matrices, the scan over a request's pieces, the outputs with norm and gate.
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

// A row of a low-rank map: sum_r w[r] x[r] (+ bias).
template <typename T>
__device__ __forceinline__ float low_rank(const T* __restrict__ w, const float* __restrict__ x, int rank) {
    float acc0 = 0.0f, acc1 = 0.0f;
    int r = 0;
    for (; r + 1 < rank; r += 2) {
        acc0 = fmaf(lb_to_float(w[r]), x[r], acc0);
        acc1 = fmaf(lb_to_float(w[r + 1]), x[r + 1], acc1);
    }
    if (r < rank) acc0 = fmaf(lb_to_float(w[r]), x[r], acc0);
    return acc0 + acc1;
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
    float acc = 0.0f;
    for (int j = 0; j < K; ++j) {
        const int back = K - 1 - j;                    // how many tokens ago
        float u = 0.0f;
        if (row - back >= row0) u = a.proj[(size_t)(row - back) * a.ld + c];
        else if (pos - back >= 0) u = ring[(size_t)((pos - back) % K) * channels + c];
        acc = fmaf(w[j], u, acc);
    }
    return acc * cm_sigmoid(acc);
}

// ---------------------------------------------------------------- row by row, from the projection to the gated heads
// Thread (c, ds) owns rows ds, ds + DS, .. of column c of the head's S (in shared memory where it fits, else where it lies).  The state travels
// before this kernel waits for the one before it.
template <typename T>
__global__ void __launch_bounds__(256) channel_memory_rows_kernel(lb_channel_memory m, StepArgs a, int ep2, int staged, int write_ring) {
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
    float* red = os + E;                       // [256]
    float* S = staged ? smem + (3 * (D + E) + 256 + 3) / 4 * 4 : st;
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

// ---------------------------------------------------------------- a low-rank map over many rows
// out[t, c] = f(sum_r x[t, r] w[c, r] + bias[c]): the decays' logarithms (base 2), or the map alone (a gate's pre-activations).  32 rows x 64 columns
// a block, a thread 2 x 4 of them.
template <typename T, bool DECAY>
__global__ void __launch_bounds__(256) low_rank_kernel(lb_channel_memory m, const float* __restrict__ x, int64_t ldx, const T* __restrict__ w, int rank,
                                                       float* __restrict__ out, int64_t ldo, int n_rows, int n_cols) {
    __shared__ float xs[32][33];
    __shared__ float ws[32][65];
    const int t0 = blockIdx.y * 32, c0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    float acc[2][4] = {};
    for (int r0 = 0; r0 < rank; r0 += 32) {
        for (int i = threadIdx.x; i < 32 * 32; i += 256) {
            const int t = i >> 5, r = i & 31;
            xs[t][r] = t0 + t < n_rows && r0 + r < rank ? x[(size_t)(t0 + t) * ldx + r0 + r] : 0.0f;
        }
        for (int i = threadIdx.x; i < 64 * 32; i += 256) {
            const int c = i >> 5, r = i & 31;
            ws[r][c] = c0 + c < n_cols && r0 + r < rank ? lb_to_float(w[(size_t)(c0 + c) * rank + r0 + r]) : 0.0f;
        }
        __syncthreads();
        const int n = min(32, rank - r0);
        for (int r = 0; r < n; ++r) {
            const float a0 = xs[ty][r], a1 = xs[ty + 16][r];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float b = ws[r][tx + 16 * j];
                acc[0][j] = fmaf(a0, b, acc[0][j]);
                acc[1][j] = fmaf(a1, b, acc[1][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty + 16 * i, c = c0 + tx + 16 * j;
            if (t >= n_rows || c >= n_cols) continue;
            float z = acc[i][j];
            if (DECAY) {
                if (m.z_bias != nullptr) z += m.z_bias[c];
                z = cm_log2_decay(m, z, c / m.dim);
            }
            out[(size_t)t * ldo + c] = z;
        }
}

// ---------------------------------------------------------------- convolution, SiLU and unit vectors over many rows
// A block per row, a warp per query, key or value head: [q | k | v] as the recurrence reads them (queries without their factor).
__global__ void __launch_bounds__(256) channel_prepare_kernel(lb_channel_memory m, StepArgs a, float* __restrict__ out, int64_t ldo) {
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const int row = blockIdx.x, seq = a.tok_seq[row], row0 = a.q_start[seq], pos = a.positions[row], channels = channels_of(m);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    const float* ring = a.state + (size_t)a.slots[seq] * m.slot_stride + (size_t)m.n_head * m.dim * m.vdim;
    for (int job = blockIdx.y * n_warps + warp; job < 2 * m.kv_head + m.n_head; job += gridDim.y * n_warps) {
        const bool is_v = job >= 2 * m.kv_head;
        const int size = is_v ? m.vdim : m.dim, first = is_v ? 2 * m.kv_head * m.dim + (job - 2 * m.kv_head) * m.vdim : job * m.dim;
        float held[8];
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = lane + 32 * i;
            held[i] = c < size ? conv_channel(m, a, ring, first + c, row, row0, pos, channels) : 0.0f;
            ss = fmaf(held[i], held[i], ss);
        }
        const float f = m.unit && !is_v ? 1.0f / sqrtf(lb_warp_sum(ss) + m.unit_eps) : 1.0f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = lane + 32 * i;
            if (c < size) out[(size_t)row * ldo + first + c] = held[i] * f;
        }
    }
}

// ---------------------------------------------------------------- pieces of 32 rows
struct PieceLayout {
    int64_t p, q, keep, b, w, u, s, total;      // floats from the start of a (piece, head)'s scratch
};
__host__ __device__ inline PieceLayout piece_layout(int D, int E, int delta) {
    auto up = [](int64_t n) { return (n + 3) / 4 * 4; };
    PieceLayout l{};
    int64_t at = 0;
    auto take = [&](int64_t n) { const int64_t r = at; at += up(n); return r; };
    l.p = take(kPiece * kPiece);                // P(t, j)
    l.q = take(kPiece * D);                     // exp(b_t) q_t
    l.keep = take(D);                           // exp(b_n)
    l.b = take(delta ? kPiece * D : 0);         // exp(b_n - b_j) k_j
    l.w = take(delta ? kPiece * D : 0);         // M K~
    l.u = take(delta ? kPiece * E : 0);         // M V; after the scan U
    l.s = take((int64_t)D * E);                 // without the delta rule the piece's own sum; after the scan the state before the piece
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

struct PieceArgs {
    const float* q;            // [T, ldq] query, key and value rows (column blocks of one buffer)
    const float* k;
    const float* v;
    int64_t ldq;
    const float* log_decay;    // [T, ldd] base 2
    int64_t ldd;
    const float* gate;         // [T, ldg] the gate's pre-activations
    int64_t ldg;
    float* scratch;            // [pieces][heads][piece_layout.total]
};

// y[t][x] = sum_j m[t][j] v[j][x] for 8 rows t0 .. t0 + 7 of one column (m [32][36] lower triangular, v column x at stride ldv).
__device__ __forceinline__ void tri_product(float (&y)[8], const float* m, const float* v, int ldv, int t0) {
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = 0.0f;
    for (int j = 0; j < t0 + 8; j += 4) {
        const float v0 = v[(size_t)j * ldv], v1 = v[(size_t)(j + 1) * ldv], v2 = v[(size_t)(j + 2) * ldv], v3 = v[(size_t)(j + 3) * ldv];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float4 r = *reinterpret_cast<const float4*>(m + (t0 + i) * 36 + j);
            y[i] = fmaf(r.x, v0, fmaf(r.y, v1, fmaf(r.z, v2, fmaf(r.w, v3, y[i]))));
        }
    }
}

template <bool DELTA>
__global__ void __launch_bounds__(256) channel_pieces_kernel(lb_channel_memory m, StepArgs a, PieceArgs w, int n_seq) {
    extern __shared__ __align__(16) float smem[];
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    int seq, piece;
    if (!find_piece(a.q_start, n_seq, blockIdx.x, &seq, &piece)) return;
    const int h = blockIdx.y, D = m.dim, E = m.vdim, LD = D + 1, LE = E + 1, g = h / (m.n_head / m.kv_head);
    const int row0 = a.q_start[seq] + piece * kPiece, n = min(kPiece, a.q_start[seq + 1] - row0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* Am = smem;                          // [32][36]
    float* M = Am + kPiece * 36;               // [32][36]
    float* beta = M + kPiece * 36;             // [32]
    float* qs = beta + kPiece;                 // [32][LD]
    float* ks = qs + kPiece * LD;              // [32][LD]
    float* bs = ks + kPiece * LD;              // [32][LD] log decays, then their running sums
    float* vs = bs + kPiece * LD;              // [32][LE]
    const PieceLayout l = piece_layout(D, E, DELTA);
    float* out = w.scratch + ((size_t)blockIdx.x * m.n_head + h) * l.total;
    for (int t = warp; t < kPiece; t += 8) {
        const bool in = t < n;
        const size_t row = (size_t)(row0 + (in ? t : 0));
        for (int d = lane; d < D; d += 32) {
            if (in) {
                cm_cp_async4(qs + t * LD + d, w.q + row * w.ldq + g * D + d);
                cm_cp_async4(ks + t * LD + d, w.k + row * w.ldq + g * D + d);
                cm_cp_async4(bs + t * LD + d, w.log_decay + row * w.ldd + h * D + d);
            } else {
                qs[t * LD + d] = ks[t * LD + d] = bs[t * LD + d] = 0.0f;
            }
        }
        for (int x = lane; x < E; x += 32) {
            if (in) cm_cp_async4(vs + t * LE + x, w.v + row * w.ldq + h * E + x);
            else vs[t * LE + x] = 0.0f;
        }
        if (DELTA && lane == 0) beta[t] = in ? cm_sigmoid(a.proj[row * a.ld + m.b_off + h]) : 0.0f;
    }
    cm_cp_commit();
    cm_cp_wait_all();
    __syncthreads();
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        float b = 0.0f;
#pragma unroll
        for (int t = 0; t < kPiece; ++t) {
            b += bs[t * LD + d];
            bs[t * LD + d] = b;
        }
    }
    __syncthreads();
    // The pairs: a warp per row t, lane j.
    for (int t = warp; t < kPiece; t += 8) {
        float p = 0.0f, av = 0.0f;
        if (lane <= t && t < n) {
            const float *qt = qs + t * LD, *kt = ks + t * LD, *bt = bs + t * LD, *kj = ks + lane * LD, *bj = bs + lane * LD;
#pragma unroll 4
            for (int d = 0; d < D; ++d) {
                const float e = exp2f(bt[d] - bj[d]) * kj[d];
                p = fmaf(qt[d], e, p);
                if (DELTA) av = fmaf(kt[d], e, av);
            }
        }
        out[l.p + t * kPiece + lane] = p * m.q_scale;
        if (DELTA) Am[t * 36 + lane] = lane < t ? av : 0.0f;
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
        const int first = DELTA ? threadIdx.x - 32 : threadIdx.x, step = DELTA ? blockDim.x - 32 : blockDim.x;
        for (int i = first; i < kPiece * D; i += step) {
            const int t = i / D, d = i - t * D;
            const float b = bs[t * LD + d], b_last = bs[(kPiece - 1) * LD + d], k = ks[t * LD + d], e = exp2f(b), kb = exp2f(b_last - b) * k;
            out[l.q + i] = qs[t * LD + d] * m.q_scale * e;
            if (DELTA) {
                out[l.b + i] = kb;
                ks[t * LD + d] = k * e;        // K~
            } else {
                ks[t * LD + d] = kb;
            }
            if (t == 0) out[l.keep + d] = exp2f(b_last);
        }
    }
    __syncthreads();
    if (DELTA) {
        // M K~ and M V: thread (column, eight rows).
        for (int i = threadIdx.x; i < 4 * (D + E); i += blockDim.x) {
            const int part = i / (D + E), x = i - part * (D + E), t0 = 8 * part;
            float y[8];
            if (x < D) tri_product(y, M, ks + x, LD, t0);
            else tri_product(y, M, vs + (x - D), LE, t0);
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                if (x < D) out[l.w + (t0 + k) * D + x] = y[k];
                else out[l.u + (t0 + k) * E + (x - D)] = y[k];
            }
        }
    } else {
        // The piece's own sum: thread (column, eight channels).
        const int parts = (D + 7) / 8;
        for (int i = threadIdx.x; i < parts * E; i += blockDim.x) {
            const int part = i / E, x = i - part * E, d0 = 8 * part;
            float y[8] = {};
            for (int j = 0; j < n; ++j) {
                const float v = vs[j * LE + x];
#pragma unroll
                for (int k = 0; k < 8; ++k) y[k] = fmaf(ks[j * LD + min(d0 + k, D - 1)], v, y[k]);
            }
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (d0 + k < D) out[l.s + (d0 + k) * E + x] = y[k];
        }
    }
}

// The scan without the delta rule: every element of S by itself, S <- exp(b_n)[d] S + sum, the state before every piece left in the sum's place.
constexpr int kAhead = 8;
__global__ void __launch_bounds__(256) channel_scan_kernel(lb_channel_memory m, StepArgs a, PieceArgs w) {
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
    float* first = w.scratch + ((size_t)g0 * m.n_head + h) * l.total;
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

// The scan under the delta rule: a block per (request, head, VT value columns) walks the request's pieces, U = M V - (M K~) S, then
// S <- exp(b_n) S + sum_j (exp(b_n - b_j) k_j) u_j^T; the next piece's matrices travel while this one is added.
template <int VT>
__global__ void __launch_bounds__(256) delta_scan_kernel(lb_channel_memory m, StepArgs a, PieceArgs w) {
    extern __shared__ __align__(16) float smem[];
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    const int seq = blockIdx.x, h = blockIdx.y, D = m.dim, E = m.vdim, c0 = blockIdx.z * VT;
    const int pieces = (a.q_start[seq + 1] - a.q_start[seq] + kPiece - 1) / kPiece;
    if (pieces <= 0) return;
    int g0 = 0;
    for (int s = 0; s < seq; ++s) g0 += (a.q_start[s + 1] - a.q_start[s] + kPiece - 1) / kPiece;
    const PieceLayout l = piece_layout(D, E, 1);
    const int LS = VT;
    const int matrix = (kPiece * D + 3) / 4 * 4, d4 = (D + 3) / 4 * 4;
    float* S = smem;                           // [d4][VT]
    float* U = S + d4 * LS;                    // [32][VT]
    float* buf = U + kPiece * VT;              // [2][W | B | keep | M V's columns]
    const int buf_floats = 2 * matrix + d4 + kPiece * VT;
    const size_t stride = (size_t)m.n_head * l.total;
    float* first = w.scratch + ((size_t)g0 * m.n_head + h) * l.total;
    float* st = a.state + (size_t)a.slots[seq] * m.slot_stride + (size_t)h * D * E;
    auto ask = [&](int p) {
        const float* src = first + (size_t)p * stride;
        float* dst = buf + (p & 1) * buf_floats;
        cm_fetch(dst, src + l.w, kPiece * D);
        cm_fetch(dst + matrix, src + l.b, kPiece * D);
        cm_fetch(dst + 2 * matrix, src + l.keep, D);
        for (int i = threadIdx.x; i < kPiece * VT; i += blockDim.x) {
            const int t = i / VT, x = i - t * VT;
            if (c0 + x < E) cm_cp_async4(dst + 2 * matrix + d4 + i, src + l.u + t * E + c0 + x);
            else dst[2 * matrix + d4 + i] = 0.0f;
        }
        cm_cp_commit();
    };
    ask(0);
    for (int i = threadIdx.x; i < d4 * VT; i += blockDim.x) {
        const int d = i / VT, x = i - d * VT;
        S[d * LS + x] = d < D && c0 + x < E ? st[(size_t)d * E + c0 + x] : 0.0f;
    }
    const int c = threadIdx.x % VT, tr = threadIdx.x / VT;
    constexpr int TR = 256 / VT;               // thread rows
    for (int p = 0; p < pieces; ++p) {
        cm_cp_wait_all();
        __syncthreads();                       // the piece has arrived; S is whole; the other buffer is free
        if (p + 1 < pieces) ask(p + 1);
        const float* W = buf + (p & 1) * buf_floats;
        const float* B = W + matrix;
        const float* keep = B + matrix;
        const float* MV = keep + d4;
        float* at = first + (size_t)p * stride;
        for (int i = threadIdx.x; i < D * VT; i += blockDim.x) {
            const int d = i / VT, x = i - d * VT;
            if (c0 + x < E) at[l.s + (size_t)d * E + c0 + x] = S[d * LS + x];
        }
        constexpr int R = kPiece / TR > 0 ? kPiece / TR : 1;
        if (tr < kPiece) {
            float y[R];
#pragma unroll
            for (int i = 0; i < R; ++i) y[i] = MV[(tr + i * TR) * VT + c];
            if ((D & 3) == 0) {
                for (int d = 0; d < D; d += 4) {
                    const float s0 = S[d * LS + c], s1 = S[(d + 1) * LS + c], s2 = S[(d + 2) * LS + c], s3 = S[(d + 3) * LS + c];
#pragma unroll
                    for (int i = 0; i < R; ++i) {
                        const float4 r = *reinterpret_cast<const float4*>(W + (tr + i * TR) * D + d);
                        y[i] = fmaf(-r.x, s0, fmaf(-r.y, s1, fmaf(-r.z, s2, fmaf(-r.w, s3, y[i]))));
                    }
                }
            } else {
                for (int d = 0; d < D; ++d) {
                    const float s = S[d * LS + c];
#pragma unroll
                    for (int i = 0; i < R; ++i) y[i] = fmaf(-W[(tr + i * TR) * D + d], s, y[i]);
                }
            }
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int t = tr + i * TR;
                U[t * VT + c] = y[i];
                if (c0 + c < E) at[l.u + (size_t)t * E + c0 + c] = y[i];
            }
        }
        __syncthreads();
        // S: thread (column, four channels at a time).
        for (int d = 4 * tr; d < D; d += 4 * TR) {
            float y[4] = {};
            if ((D & 3) == 0) {
#pragma unroll 8
                for (int t = 0; t < kPiece; ++t) {
                    const float u = U[t * VT + c];
                    const float4 r = *reinterpret_cast<const float4*>(B + t * D + d);
                    y[0] = fmaf(r.x, u, y[0]);
                    y[1] = fmaf(r.y, u, y[1]);
                    y[2] = fmaf(r.z, u, y[2]);
                    y[3] = fmaf(r.w, u, y[3]);
                }
            } else {
                for (int t = 0; t < kPiece; ++t) {
                    const float u = U[t * VT + c];
#pragma unroll
                    for (int k = 0; k < 4; ++k) y[k] = fmaf(B[t * D + min(d + k, D - 1)], u, y[k]);
                }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (d + k < D) S[(d + k) * LS + c] = fmaf(keep[d + k], S[(d + k) * LS + c], y[k]);
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < D * VT; i += blockDim.x) {
        const int d = i / VT, x = i - d * VT;
        if (c0 + x < E) st[(size_t)d * E + c0 + x] = S[d * LS + x];
    }
}

// The outputs of a piece with the heads' norm and gate.  Thread (c, tg) owns column c for the R rows tg R .. tg R + R - 1.
template <typename T, int R, bool DELTA>
__global__ void __launch_bounds__(256) channel_outputs_kernel(lb_channel_memory m, StepArgs a, PieceArgs w, int n_seq) {
    extern __shared__ __align__(16) float smem[];
    constexpr int EP = 8 * R;                  // threads across the columns: 256 / (32 / R)
    lb_wait_for_predecessor();
    lb_dependents_may_launch();
    int seq, piece;
    if (!find_piece(a.q_start, n_seq, blockIdx.x, &seq, &piece)) return;
    const int h = blockIdx.y, D = m.dim, E = m.vdim, d4 = (D + 3) / 4 * 4;
    const int row0 = a.q_start[seq] + piece * kPiece, n = min(kPiece, a.q_start[seq + 1] - row0);
    float* P = smem;                           // [32][32]
    float* qs = P + kPiece * kPiece;           // [32][d4]
    float* os = qs + kPiece * d4;              // [32][E + 1]
    const PieceLayout l = piece_layout(D, E, DELTA);
    const float* in = w.scratch + ((size_t)blockIdx.x * m.n_head + h) * l.total;
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
    cm_cp_commit();
    cm_cp_wait_all();
    __syncthreads();
    const int c = threadIdx.x % EP, t0 = threadIdx.x / EP * R;
    if (c < E) {
        float y[R];
#pragma unroll
        for (int i = 0; i < R; ++i) y[i] = 0.0f;
        const float* S = in + l.s + c;
        for (int d = 0; d < D; d += 4) {
            float s[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) s[k] = d + k < D ? S[(size_t)(d + k) * E] : 0.0f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const float4 q = *reinterpret_cast<const float4*>(qs + (t0 + i) * d4 + d);
                y[i] = fmaf(q.x, s[0], fmaf(q.y, s[1], fmaf(q.z, s[2], fmaf(q.w, s[3], y[i]))));
            }
        }
        const float* u = DELTA ? in + l.u + c : w.v + (size_t)row0 * w.ldq + h * E + c;
        const size_t ldu = DELTA ? (size_t)E : (size_t)w.ldq;
        const int last = min(n, t0 + R);       // rows after the last of this thread's are not seen
        for (int j = 0; j < last; j += 4) {
            float s[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) s[k] = j + k < n ? u[(size_t)(j + k) * ldu] : 0.0f;
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
        const float inv = 1.0f / sqrtf(lb_warp_sum(ss) / (float)E + m.eps);
        const size_t row = (size_t)(row0 + t);
        for (int x = lane; x < E; x += 32) {
            if (a.o != nullptr) a.o[row * a.ldo + h * E + x] = o[x];
            static_cast<T*>(a.heads)[row * a.ldh + h * E + x] = lb_from_float<T>(o[x] * inv * m.norm[x] * cm_gate(w.gate[row * w.ldg + h * E + x], m.gate_act));
        }
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
    const size_t base = (3 * ((size_t)m.dim + m.vdim) + 256 + 3) / 4 * 4 * sizeof(float), with_state = base + (size_t)m.dim * m.vdim * sizeof(float);
    const int staged = with_state <= 160 * 1024 ? 1 : 0;
    const size_t smem = staged ? with_state : base;
    auto launch = [&](auto kernel) -> int {
        if (smem > 48 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, dim3(n_seq, m.n_head), dim3(256), smem, s, m, a, ep2, staged, decode_only));
        return LB_OK;
    };
    if (int rc = dtype == LB_F32 ? launch(channel_memory_rows_kernel<float>) : launch(channel_memory_rows_kernel<__nv_bfloat16>)) return rc;
    if (m.conv != nullptr && !decode_only) return launch_ring(m, a, n_seq, s);
    return LB_OK;
}

extern "C" int64_t lb_channel_memory_pieces_floats(int n_tokens, int n_seq, int n_head, int dim, int vdim, int delta) {
    return ((int64_t)n_tokens / kPiece + n_seq) * n_head * piece_layout(dim, vdim, delta).total;
}

extern "C" int lb_channel_memory_pieces(int dtype, const lb_channel_memory* memory, const lb_channel_step* step, float* rows, float* log_decay, float* gate,
                                        float* scratch, int n_tokens, int n_seq, void* stream) {
    if (int rc = check_shape(memory)) return rc;
    LB_CHECK_ARG(dtype == LB_F32 || dtype == LB_BF16, "channel memory: unknown dtype %d", dtype);
    LB_CHECK_ARG(scratch != nullptr && log_decay != nullptr && ((memory->conv == nullptr && !memory->unit) || rows != nullptr) && (memory->g2 == nullptr || gate != nullptr),
                 "channel memory in pieces: scratch is missing");
    if (n_seq == 0 || n_tokens == 0) return LB_OK;
    const lb_channel_memory m = *memory;
    const StepArgs a = step_of(step);
    auto s = static_cast<cudaStream_t>(stream);
    const int QD = m.kv_head * m.dim, HD = m.n_head * m.dim, HE = m.n_head * m.vdim, channels = 2 * QD + HE;
    const dim3 tiles_d((HD + 63) / 64, (n_tokens + 31) / 32), tiles_e((HE + 63) / 64, (n_tokens + 31) / 32);
    // The low-rank maps.
    if (dtype == LB_F32) {
        LB_CHECK_CUDA(lb_launch_overlapped(low_rank_kernel<float, true>, tiles_d, dim3(256), 0, s, m, a.proj + m.a_off, a.ld, (const float*)m.a2, m.rank, log_decay,
                                           (int64_t)HD, n_tokens, HD));
        if (m.g2 != nullptr)
            LB_CHECK_CUDA(lb_launch_overlapped(low_rank_kernel<float, false>, tiles_e, dim3(256), 0, s, m, a.proj + m.g_off, a.ld, (const float*)m.g2, m.gate_rank,
                                               gate, (int64_t)HE, n_tokens, HE));
    } else {
        LB_CHECK_CUDA(lb_launch_overlapped(low_rank_kernel<__nv_bfloat16, true>, tiles_d, dim3(256), 0, s, m, a.proj + m.a_off, a.ld, (const __nv_bfloat16*)m.a2,
                                           m.rank, log_decay, (int64_t)HD, n_tokens, HD));
        if (m.g2 != nullptr)
            LB_CHECK_CUDA(lb_launch_overlapped(low_rank_kernel<__nv_bfloat16, false>, tiles_e, dim3(256), 0, s, m, a.proj + m.g_off, a.ld,
                                               (const __nv_bfloat16*)m.g2, m.gate_rank, gate, (int64_t)HE, n_tokens, HE));
    }
    PieceArgs w{};
    w.q = a.proj; w.ldq = a.ld;
    if (m.conv != nullptr || m.unit) {
        const int jobs = 2 * m.kv_head + m.n_head;
        LB_CHECK_CUDA(lb_launch_overlapped(channel_prepare_kernel, dim3(n_tokens, (jobs + 7) / 8), dim3(256), 0, s, m, a, rows, (int64_t)channels));
        w.q = rows;
        w.ldq = channels;
        if (m.conv != nullptr)
            if (int rc = launch_ring(m, a, n_seq, s)) return rc;
    }
    w.k = w.q + QD;
    w.v = w.q + 2 * QD;
    w.log_decay = log_decay;
    w.ldd = HD;
    w.gate = m.g2 != nullptr ? gate : a.proj + m.g_off;
    w.ldg = m.g2 != nullptr ? HE : a.ld;
    w.scratch = scratch;
    const int pieces = n_tokens / kPiece + n_seq, D = m.dim, E = m.vdim, d4 = (D + 3) / 4 * 4;
    auto launch = [&](auto kernel, dim3 grid, size_t smem, auto... args) -> int {
        LB_CHECK_ARG(smem <= 220 * 1024, "channel memory in pieces: heads of %d x %d values do not fit shared memory", D, E);
        if (smem > 48 * 1024) LB_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LB_CHECK_CUDA(lb_launch_overlapped(kernel, grid, dim3(256), smem, s, args...));
        return LB_OK;
    };
    const size_t own = (2 * kPiece * 36 + kPiece + 3 * (size_t)kPiece * (D + 1) + (size_t)kPiece * (E + 1)) * sizeof(float);
    constexpr int VT = 16;
    if (m.delta) {
        if (int rc = launch(channel_pieces_kernel<true>, dim3(pieces, m.n_head), own, m, a, w, n_seq)) return rc;
        const size_t scan = ((size_t)d4 * VT + kPiece * VT + 2 * (2 * (size_t)kPiece * d4 + d4 + kPiece * VT)) * sizeof(float);
        if (int rc = launch(delta_scan_kernel<VT>, dim3(n_seq, m.n_head, (E + VT - 1) / VT), scan, m, a, w)) return rc;
    } else {
        if (int rc = launch(channel_pieces_kernel<false>, dim3(pieces, m.n_head), own, m, a, w, n_seq)) return rc;
        if (int rc = launch(channel_scan_kernel, dim3(n_seq, m.n_head, (D * E + 255) / 256), 0, m, a, w)) return rc;
    }
    const size_t outs = (kPiece * kPiece + (size_t)kPiece * d4 + (size_t)kPiece * (E + 1)) * sizeof(float);
    const dim3 grid(pieces, m.n_head);
#define LB_OUTPUTS(T, DELTA)                                                                             \
    (E <= 8     ? launch(channel_outputs_kernel<T, 1, DELTA>, grid, outs, m, a, w, n_seq)                \
     : E <= 16  ? launch(channel_outputs_kernel<T, 2, DELTA>, grid, outs, m, a, w, n_seq)                \
     : E <= 32  ? launch(channel_outputs_kernel<T, 4, DELTA>, grid, outs, m, a, w, n_seq)                \
     : E <= 64  ? launch(channel_outputs_kernel<T, 8, DELTA>, grid, outs, m, a, w, n_seq)                \
     : E <= 128 ? launch(channel_outputs_kernel<T, 16, DELTA>, grid, outs, m, a, w, n_seq)               \
                : launch(channel_outputs_kernel<T, 32, DELTA>, grid, outs, m, a, w, n_seq))
    if (dtype == LB_F32) return m.delta ? LB_OUTPUTS(float, true) : LB_OUTPUTS(float, false);
    return m.delta ? LB_OUTPUTS(__nv_bfloat16, true) : LB_OUTPUTS(__nv_bfloat16, false);
#undef LB_OUTPUTS
}
