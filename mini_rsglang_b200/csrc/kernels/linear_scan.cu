// Recurrences that are linear in their state, a matrix S [d, e] per (request, head):
//
//     S_t = keep_t S_(t-1) + take_t k_t v_t^T,   o_t = S_t^T q_t          (and with a normaliser n_t likewise with k alone, c_t = n_t . q_t)
//
// keep is a constant a head (a retention: take = 1), comes a token with take (gates of an exponential memory), or is one number
// a token and key channel, which then acts on the rows of S (a gated linear attention: take = 1).  Everything here is float32.  S (and n) live in the request's state slot between steps; where a sequence starts at position 0 its
// state counts as zero, whatever the slot held (slots are used again).  State slot -1: a padding sequence, nothing is read or
// written.  The step's facts come from device arrays only, so a step can be recorded.
//
//   rotate_heads       q and k heads inside the float32 projection turn by their token's position, in place
//   memory_gates       keep, take and exp(-m) of every (token, head) from the raw gates of an exponential memory with a running
//                      maximum m (which starts at 0)
//   linear_scan        the recurrence (linear_step: the same for decoded tokens)
//   channel_fold       keeps a key channel from two thin products, folded into k and q so that the recurrence itself meets none
//   narrow_columns     a range of float32 columns as rows of the engine's dtype
#include "common.cuh"
#include "pairs.cuh"

namespace {

// ---------------------------------------------------------------------------------------------
// rows [tokens, stride] float32; `heads` heads of d elements from column `offset` on; the first `rot` elements of a head turn:
// element i with i + rot / 2 by the step's table [tokens, rot / 2, 2] of cosines and sines.  VEC: four pairs a thread.
// ---------------------------------------------------------------------------------------------
template <bool VEC>
__global__ void rotate_heads_kernel(float* __restrict__ rows, int stride, int offset, const float* __restrict__ table, int tokens,
                                    int heads, int d, int rot) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int half = rot / 2;
    float* row = rows + t * stride + offset;
    const float* turn = table + t * (size_t)rot;
    if (VEC) {
        const int quads = half >> 2;
        for (int at = threadIdx.x; at < heads * quads; at += blockDim.x) {
            const int i = (at % quads) * 4;
            float* x = row + (size_t)(at / quads) * d + i;
            const float4 c01 = *reinterpret_cast<const float4*>(turn + 2 * i), c23 = *reinterpret_cast<const float4*>(turn + 2 * i + 4);
            const float4 u = *reinterpret_cast<const float4*>(x), v = *reinterpret_cast<const float4*>(x + half);
            *reinterpret_cast<float4*>(x) = make_float4(u.x * c01.x - v.x * c01.y, u.y * c01.z - v.y * c01.w, u.z * c23.x - v.z * c23.y,
                                                        u.w * c23.z - v.w * c23.w);
            *reinterpret_cast<float4*>(x + half) = make_float4(v.x * c01.x + u.x * c01.y, v.y * c01.z + u.y * c01.w,
                                                               v.z * c23.x + u.z * c23.y, v.w * c23.z + u.w * c23.w);
        }
    } else {
        for (int at = threadIdx.x; at < heads * half; at += blockDim.x) {
            const int i = at % half;
            float* x = row + (size_t)(at / half) * d + i;
            const float c = turn[2 * i], s = turn[2 * i + 1], u = x[0], v = x[half];
            x[0] = u * c - v * s;
            x[half] = v * c + u * s;
        }
    }
}

template <typename T>
__global__ void narrow_columns_kernel(const float* __restrict__ rows, int stride, int offset, T* __restrict__ out, long long total, int columns,
                                      int live) {
    pdl_launch_dependents();
    pdl_wait();
    for (long long at = (long long)blockIdx.x * blockDim.x + threadIdx.x; at < total; at += (long long)gridDim.x * blockDim.x) {
        const long long t = at / columns;
        const int c = (int)(at % columns);
        out[at] = from_float<T>(c < live ? rows[t * stride + offset + c] : 0.0f);
    }
}

// ---------------------------------------------------------------------------------------------
// Gates of an exponential memory.  Per head: i = cap tanh((raw_i + bias_i) / cap), f = logsigmoid(cap tanh((raw_f + bias_f) / cap)),
// m_t = max(f_t + m_(t-1), i_t); keep_t = exp(f_t + m_(t-1) - m_t), take_t = exp(i_t - m_t), floor_t = exp(-m_t).
// One block a (sequence, head); a block's worth of tokens at a time by a scan over the maps m -> max(A + m, B), whose
// composition is (A1, B1) then (A2, B2) = (A1 + A2, max(B1 + A2, B2)).  coef [tokens, 3 heads]: keep | take | floor.
// ---------------------------------------------------------------------------------------------
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.0f) - log1pf(expf(-fabsf(x))); }

__global__ void memory_gates_kernel(const float* __restrict__ raw, int raw_stride, int i_offset, int f_offset,
                                    const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap,
                                    float* __restrict__ m_state, long long state_stride, const int* __restrict__ positions,
                                    const int* __restrict__ q_start, const int* __restrict__ state_slots, float* __restrict__ coef,
                                    int heads, int write_state) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float total_a[32], total_b[32], carried;
    const int seq = blockIdx.x, head = blockIdx.y;
    const int first = q_start[seq], last = q_start[seq + 1];
    const int slot = state_slots[seq];
    if (slot < 0 || last <= first) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* mine = m_state + (long long)slot * state_stride + head;
    float m0 = positions[first] == 0 ? 0.0f : *mine;
    const float bi = i_bias[head], bf = f_bias[head];
    for (int base = first; base < last; base += blockDim.x) {
        const int t = base + threadIdx.x;
        const bool live = t < last;
        float in = 0.0f, keep = 0.0f;
        if (live) {
            const float* r = raw + (size_t)t * raw_stride;
            in = cap * tanhf((r[i_offset + head] + bi) / cap);
            keep = log_sigmoid_f(cap * tanhf((r[f_offset + head] + bf) / cap));
        }
        float a = live ? keep : 0.0f, b = live ? in : -CUDART_INF_F;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float a1 = __shfl_up_sync(0xffffffffu, a, o), b1 = __shfl_up_sync(0xffffffffu, b, o);
            if (lane >= o) {
                b = fmaxf(b1 + a, b);
                a += a1;
            }
        }
        if (lane == 31) total_a[warp] = a, total_b[warp] = b;
        __syncthreads();
        float before = m0;                                   // m ahead of this warp's first token
        for (int w = 0; w < warp; ++w) before = fmaxf(total_a[w] + before, total_b[w]);
        const float m = fmaxf(a + before, b);
        float previous = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) previous = before;
        if (live) {
            float* c = coef + (size_t)t * 3 * heads + head;
            c[0] = expf(keep + previous - m);
            c[heads] = expf(in - m);
            c[2 * heads] = expf(-m);
            if (t == last - 1 || threadIdx.x == blockDim.x - 1) carried = m;
        }
        __syncthreads();
        m0 = carried;
    }
    if (write_state && threadIdx.x == 0) *mine = m0;
}

// ---------------------------------------------------------------------------------------------
// The recurrence.  A thread keeps SCAN_ROWS rows x 4 neighbouring columns of S in registers, two rows to a 64-bit register
// pair, so that one instruction (fma.rn.f32x2, two independent float32 multiply-adds) serves two rows; the PARTS lanes that
// share four columns cover the d rows, so what a thread reads of k and q from shared memory serves four columns, and a
// token's read-out is a reduction that hands its columns out while it sums (2 + 1 + 1 ... shuffles).  The tokens' k, q and v
// come through two stages of shared memory, filled by cp.async a batch ahead.
//
// The decay costs no instruction an element: with P the product of the keeps since S was last rescaled, the registers hold
// S / P, a token adds (take / P) k v^T and its read-out is P (S / P)^T q.  A batch's prefix products are made by one warp a
// batch ahead; where P would fall below SCAN_LEAST within a batch the registers are first multiplied by it and P starts
// again at 1, and a batch whose own product falls below it is walked with the decay applied token by token.
//
// SCAN_WHOLE: a sequence's rows in one go, from the slot's state to the slot's state.  Long portions of few sequences are cut
// into chunks of `chunk_len` rows that run side by side: SCAN_LOCAL runs every chunk from zero and leaves its end state and
// the product of its keeps in scratch, scan_chunk_states walks a sequence's chunks once and turns the end states into the
// state at every chunk's start (and the slot's new state), SCAN_FINAL runs every chunk from there and writes o.
// ---------------------------------------------------------------------------------------------
#define SCAN_ROWS 16
#define SCAN_PITCH (SCAN_ROWS + 4)       // 16-byte reads of the parts fall on different banks
#define SCAN_LEAST 1e-8f
#define SCAN_BATCH 8                     // tokens a batch, at most
enum { SCAN_WHOLE = 0, SCAN_LOCAL = 1, SCAN_FINAL = 2 };

struct ScanArgs {
    const float *q, *k, *v;              // columns of float32 rows of `stride` floats; heads of d, d and e elements
    int stride;
    const float* decay;                  // [heads], or null: the coefficients
    const float* coef;                   // [tokens, coef_stride]: keep of every head, then take; keeps lie in 0 .. 1
    int coef_stride;
    float* state;                        // [slots][heads, d, e]
    float* norm_state;                   // [slots][heads, d], or null: no normaliser
    long long state_stride;
    const int *positions, *q_start, *state_slots;
    float* out;                          // [tokens, heads * e]
    float* norm_out;                     // [tokens, heads]
    int heads, d, e, cols, slices, batch, write_state, vec_qk, vec_v, vec_state, vec_out;
    float *chunk_state, *chunk_decay;
    int chunk_len, max_chunks, chunk_floats;
    // keeps a key channel (CHANNEL); rows of a batch are then counted from the step's first row, and so are those of a chunk
    float* keeps;                        // [tokens, heads * d]: what channel_fold leaves
    int* direct;                         // [batches, heads]: the batch's keeps are applied token by token
    int vec_keeps;
    // what a decoded token's keeps are made of
    const float* low;                    // a column range of the float32 rows: the first thin product, `rank` wide
    const void* up;                      // [heads * d, rank], float32 or bfloat16: the second
    const float* keep_bias;              // [heads * d]
    float inverse_tau;
    int rank;
};

// sigmoid(z)^(1 / tau)
__device__ __forceinline__ float channel_keep(float z, float inverse_tau) { return expf(log_sigmoid_f(z) * inverse_tau); }

// ---------------------------------------------------------------------------------------------
// Keeps a key channel: a_t = sigmoid(up low_t + bias)^(1 / tau), [heads * d] a token.  The decay acts on the rows of S, so with P_t
// a channel's product of keeps since its batch (of `batch` rows, counted from the step's first row) or its sequence began,
// S_t = diag(P_t) U_t with U_t = U_(t-1) + (k_t / P_t) v_t^T and o_t = U_t^T (P_t q_t): k and q are divided and multiplied in place,
// P goes to `keeps`, and the recurrence multiplies S by P once a batch.  Where some P of a (batch, head) falls below FOLD_LEAST
// nothing is folded there: `keeps` gets the keeps themselves and `direct` says so.
// A thread takes a channel and the rows of a batch; a block whole heads.  Dynamic shared memory: SCAN_BATCH * rank floats.
// ---------------------------------------------------------------------------------------------
#define FOLD_LEAST 1e-15f
template <typename W>
__global__ void channel_fold_kernel(const ScanArgs A, float* __restrict__ q, float* __restrict__ k, const int* __restrict__ seq_of_token,
                                    int tokens, int heads_a_block) {
    extern __shared__ __align__(16) float low_rows[];
    __shared__ int small[32];
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * A.batch, n = min(A.batch, tokens - t0);
    const int head0 = blockIdx.y * heads_a_block, own = threadIdx.x / A.d;
    const bool live = own < heads_a_block && head0 + own < A.heads;
    const int channel = head0 * A.d + threadIdx.x;
    float a[SCAN_BATCH], P[SCAN_BATCH], qs[SCAN_BATCH], ks[SCAN_BATCH];
#pragma unroll
    for (int j = 0; j < SCAN_BATCH; ++j) {                   // asked for ahead of their use
        const bool here = live && j < n;
        qs[j] = here ? q[(size_t)(t0 + j) * A.stride + channel] : 0.0f;
        ks[j] = here ? k[(size_t)(t0 + j) * A.stride + channel] : 0.0f;
    }
    for (int i = threadIdx.x; i < SCAN_BATCH * A.rank; i += blockDim.x) {        // [rank][SCAN_BATCH]
        const int j = i / A.rank, r = i % A.rank;
        low_rows[r * SCAN_BATCH + j] = j < n ? A.low[(size_t)(t0 + j) * A.stride + r] : 0.0f;
    }
    if (threadIdx.x < 32) small[threadIdx.x] = 0;
    __syncthreads();
    if (live) {
        const float b = A.keep_bias[channel];
#pragma unroll
        for (int j = 0; j < SCAN_BATCH; ++j) a[j] = b;
        const W* up = (const W*)A.up + (size_t)channel * A.rank;
        auto add = [&](float w, int r) {
            const float4 lo = *reinterpret_cast<const float4*>(low_rows + r * SCAN_BATCH), hi = *reinterpret_cast<const float4*>(low_rows + r * SCAN_BATCH + 4);
            a[0] = fmaf(w, lo.x, a[0]), a[1] = fmaf(w, lo.y, a[1]), a[2] = fmaf(w, lo.z, a[2]), a[3] = fmaf(w, lo.w, a[3]);
            a[4] = fmaf(w, hi.x, a[4]), a[5] = fmaf(w, hi.y, a[5]), a[6] = fmaf(w, hi.z, a[6]), a[7] = fmaf(w, hi.w, a[7]);
        };
        constexpr int PIECE = 16 / sizeof(W);                // matrix elements of a 16-byte load
        if (A.rank % PIECE == 0 && ((uintptr_t)A.up & 15) == 0) {
            for (int r = 0; r < A.rank; r += PIECE) {
                const uint4 raw = *reinterpret_cast<const uint4*>(up + r);
                const W* w = reinterpret_cast<const W*>(&raw);
#pragma unroll
                for (int u = 0; u < PIECE; ++u) add(to_float(w[u]), r + u);
            }
        } else {
            for (int r = 0; r < A.rank; ++r) add(to_float(up[r]), r);
        }
        float p = 1.0f;
        bool tiny = false;
        int before = -1;
#pragma unroll
        for (int j = 0; j < SCAN_BATCH; ++j) {
            if (j >= n) continue;
            const int seq = seq_of_token[t0 + j];
            if (seq != before) p = 1.0f;
            before = seq;
            a[j] = channel_keep(a[j], A.inverse_tau);
            p *= a[j];
            P[j] = p;
            tiny = tiny || p < FOLD_LEAST;
        }
        if (tiny) small[own] = 1;
    }
    __syncthreads();
    if (!live) return;
    const bool direct = small[own];
#pragma unroll
    for (int j = 0; j < SCAN_BATCH; ++j) {
        if (j >= n) continue;
        const size_t t = t0 + j;
        A.keeps[t * A.heads * A.d + channel] = direct ? a[j] : P[j];
        if (!direct) {
            k[t * A.stride + channel] = ks[j] / P[j];
            q[t * A.stride + channel] = qs[j] * P[j];
        }
    }
    if (threadIdx.x % A.d == 0) A.direct[(size_t)blockIdx.x * A.heads + head0 + own] = direct;
}

__device__ __forceinline__ void scan_copy16(float* to, const float* from) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(to)), "l"(from));
}
__device__ __forceinline__ void scan_copy4(float* to, const float* from) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(to)), "l"(from));
}

template <int MODE, int PARTS, bool CHANNEL>
__global__ void __launch_bounds__(256, 2) linear_scan_kernel(const ScanArgs A) {
    extern __shared__ __align__(16) float stage[];
    __shared__ __align__(16) float4 facts[2][SCAN_BATCH];    // of a token: take / p, p, keep, take; p the batch's product of keeps so far
    constexpr int GROUPS = 32 / PARTS;                       // groups of four columns a warp covers
    constexpr int VECTOR = PARTS * SCAN_PITCH;               // floats of a k (or q) in shared memory
    constexpr int PAIRS = SCAN_ROWS / 2;
    constexpr bool PRODUCTS = CHANNEL && MODE == SCAN_LOCAL;
    __shared__ float products[PRODUCTS ? PARTS * SCAN_ROWS : 1];     // of the chunk's keeps, a channel each; one warp's alone
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int token_floats = 2 * VECTOR + A.cols, stage_floats = A.batch * token_floats + (CHANNEL ? VECTOR : 0);
    for (int i = threadIdx.x; i < 2 * stage_floats; i += blockDim.x) stage[i] = 0.0f;      // rows beyond d, columns beyond e
    if (PRODUCTS)
        for (int i = threadIdx.x; i < PARTS * SCAN_ROWS; i += blockDim.x) products[i] = 1.0f;
    __syncthreads();
    pdl_wait();
    const int seq = blockIdx.x, head = blockIdx.y / A.slices, slice = blockIdx.y % A.slices, chunk = blockIdx.z;
    const int seq_first = A.q_start[seq], seq_last = A.q_start[seq + 1];
    const int slot = A.state_slots[seq];
    if (slot < 0 || seq_last <= seq_first) return;
    const int chunk_first = MODE == SCAN_WHOLE ? 0 : ((CHANNEL ? seq_first / A.chunk_len : 0) + chunk) * A.chunk_len + (CHANNEL ? 0 : seq_first);
    const int first = MODE == SCAN_WHOLE ? seq_first : max(seq_first, chunk_first);
    const int last = MODE == SCAN_WHOLE ? seq_last : min(seq_last, chunk_first + A.chunk_len);
    if (first >= last) return;
    const int part = lane / GROUPS, place = (warp * GROUPS + lane % GROUPS) * 4, col = slice * A.cols + place;
    const int row0 = part * SCAN_ROWS;
    // a normaliser is one more column behind S's (at a multiple of four), whose value is always 1
    const int norm_col = A.norm_state ? (A.e + 3) / 4 * 4 : -4;
    const bool is_norm = col == norm_col;
    const bool idle = slice * A.cols + warp * GROUPS * 4 >= max(A.e, norm_col + 4);      // a warp without columns
    const size_t chunk_at = (((size_t)seq * A.heads + head) * A.max_chunks + chunk);
    float* mine = MODE == SCAN_WHOLE ? A.state + (long long)slot * A.state_stride + (size_t)head * A.d * A.e : A.chunk_state + chunk_at * A.chunk_floats;
    float* norm_mine = MODE == SCAN_WHOLE ? A.norm_state + (long long)slot * A.state_stride + (size_t)head * A.d : mine + (size_t)A.d * A.e;
    const bool zero = MODE == SCAN_LOCAL || (MODE == SCAN_WHOLE && A.positions[seq_first] == 0);

    const int q_at = head * A.d, v_at = head * A.e + slice * A.cols, live_cols = min(A.cols, A.e - slice * A.cols);
    auto issue = [&](int t0, int n, int buffer) {
        float* base = stage + buffer * stage_floats;
        for (int j = warp; j < n; j += warps) {              // a warp copies a token
            float* to = base + j * token_floats;
            const size_t row = (size_t)(t0 + j) * A.stride;
            if (A.vec_qk) {
                for (int i = 4 * lane; i < A.d; i += 128) {
                    const int where = (i / SCAN_ROWS) * SCAN_PITCH + i % SCAN_ROWS;
                    scan_copy16(to + where, A.k + row + q_at + i);
                    if (MODE != SCAN_LOCAL) scan_copy16(to + VECTOR + where, A.q + row + q_at + i);
                }
            } else {
                for (int i = lane; i < A.d; i += 32) {
                    const int where = (i / SCAN_ROWS) * SCAN_PITCH + i % SCAN_ROWS;
                    scan_copy4(to + where, A.k + row + q_at + i);
                    if (MODE != SCAN_LOCAL) scan_copy4(to + VECTOR + where, A.q + row + q_at + i);
                }
            }
            if (A.vec_v) {
                for (int i = 4 * lane; i < live_cols; i += 128) scan_copy16(to + 2 * VECTOR + i, A.v + row + v_at + i);
            } else {
                for (int i = lane; i < live_cols; i += 32) scan_copy4(to + 2 * VECTOR + i, A.v + row + v_at + i);
            }
        }
        if (CHANNEL && warp == warps - 1) {                  // what S is multiplied by behind the batch
            const float* from = A.keeps + (size_t)(t0 + n - 1) * A.heads * A.d + q_at;
            float* to = base + A.batch * token_floats;
            if (A.vec_keeps) {
                for (int i = 4 * lane; i < A.d; i += 128) scan_copy16(to + (i / SCAN_ROWS) * SCAN_PITCH + i % SCAN_ROWS, from + i);
            } else {
                for (int i = lane; i < A.d; i += 32) scan_copy4(to + (i / SCAN_ROWS) * SCAN_PITCH + i % SCAN_ROWS, from + i);
            }
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    // rows of the batch that begins at row t
    auto rows_at = [&](int t) { return min(CHANNEL ? A.batch - t % A.batch : A.batch, last - t); };
    auto direct_at = [&](int t) { return CHANNEL && A.direct[(size_t)(t / A.batch) * A.heads + head] != 0; };
    const float fixed = A.decay ? A.decay[head] : 1.0f;
    auto read_facts = [&](int t0, int n) {                   // keep and take of token t0 + lane, warp 0
        if (A.decay || lane >= n) return make_float2(lane < n ? fixed : 1.0f, 1.0f);
        const float* c = A.coef + (size_t)(t0 + lane) * A.coef_stride + head;
        return make_float2(c[0], c[A.heads]);
    };
    auto write_facts = [&](float2 raw, int buffer) {
        float p = raw.x;
#pragma unroll
        for (int o = 1; o < SCAN_BATCH; o <<= 1) {
            const float before = __shfl_up_sync(0xffffffffu, p, o);
            if (lane >= o) p *= before;
        }
        if (lane < A.batch) facts[buffer][lane] = make_float4(raw.y / p, p, raw.x, raw.y);
    };
    issue(first, rows_at(first), 0);
    if (!CHANNEL && warp == 0) write_facts(read_facts(first, rows_at(first)), 0);
    bool direct = direct_at(first);

    pair s[4][PAIRS];                                        // a column's rows two by two
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
        float x[4][2] = {{0.0f, 0.0f}, {0.0f, 0.0f}, {0.0f, 0.0f}, {0.0f, 0.0f}};
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int row = row0 + 2 * i + u;
            if (zero || row >= A.d) continue;
            const float* from = mine + (size_t)row * A.e + col;
            if (A.vec_state) {
                if (col < A.e) {
                    const float4 f = *reinterpret_cast<const float4*>(from);
                    x[0][u] = f.x, x[1][u] = f.y, x[2][u] = f.z, x[3][u] = f.w;
                }
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (col + c < A.e) x[c][u] = from[c];
            }
            if (is_norm) x[0][u] = norm_mine[row];
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) s[c][i] = make_pair(x[c][0], x[c][1]);
    }
    auto rescale = [&](float by) {
        const pair f = make_pair(by, by);
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
#pragma unroll
            for (int c = 0; c < 4; ++c) s[c][i] = mul2(s[c][i], f);
        }
    };
    // one token: `weight` multiplies what is added, `factor` what is read
    float* to = A.out + (size_t)first * A.heads * A.e + (size_t)head * A.e + col;
    if (is_norm) to = A.norm_out + (size_t)first * A.heads + head;
    const size_t out_step = is_norm ? A.heads : (size_t)A.heads * A.e;
    const int live = is_norm ? 1 : A.e - col;                // columns of these four that are there
    auto walk = [&](const float* token, float weight, float factor) {
        float4 vv = *reinterpret_cast<const float4*>(token + 2 * VECTOR + place);
        if (is_norm) vv.x = 1.0f;                            // the columns behind e are zero
        const pair tv[4] = {make_pair(vv.x * weight, vv.x * weight), make_pair(vv.y * weight, vv.y * weight),
                            make_pair(vv.z * weight, vv.z * weight), make_pair(vv.w * weight, vv.w * weight)};
        pair y[4];
        const float* kp = token + part * SCAN_PITCH;
#pragma unroll
        for (int i = 0; i < PAIRS; i += 2) {
            const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(kp + 2 * i);
            ulonglong2 qq = make_ulonglong2(0ull, 0ull);
            if (MODE != SCAN_LOCAL) qq = *reinterpret_cast<const ulonglong2*>(kp + VECTOR + 2 * i);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                s[c][i] = fma2(kk.x, tv[c], s[c][i]);
                s[c][i + 1] = fma2(kk.y, tv[c], s[c][i + 1]);
                if (MODE != SCAN_LOCAL) {
                    y[c] = i == 0 ? mul2(s[c][i], qq.x) : fma2(s[c][i], qq.x, y[c]);
                    y[c] = fma2(s[c][i + 1], qq.y, y[c]);
                }
            }
        }
        if (MODE == SCAN_LOCAL) return;
        const float z[4] = {both(y[0]), both(y[1]), both(y[2]), both(y[3])};
        if (PARTS == 1) {
            if (A.vec_out && !is_norm) {
                if (live > 0) *reinterpret_cast<float4*>(to) = make_float4(z[0] * factor, z[1] * factor, z[2] * factor, z[3] * factor);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (c < live) to[c] = z[c] * factor;
            }
            return;
        }
        const bool upper = part & 1;                         // this lane goes on with the upper two of the four columns
        float z0 = upper ? z[2] : z[0], z1 = upper ? z[3] : z[1];
        z0 += __shfl_xor_sync(0xffffffffu, upper ? z[0] : z[2], GROUPS);
        z1 += __shfl_xor_sync(0xffffffffu, upper ? z[1] : z[3], GROUPS);
        const int at = upper ? 2 : 0;
        if (PARTS == 2) {
            if (at < live) to[at] = z0 * factor;
            if (at + 1 < live) to[at + 1] = z1 * factor;
            return;
        }
        const bool second = part & 2;
        float one = second ? z1 : z0;
        one += __shfl_xor_sync(0xffffffffu, second ? z0 : z1, 2 * GROUPS);
#pragma unroll
        for (int o = 4 * GROUPS; o < 32; o <<= 1) one += __shfl_xor_sync(0xffffffffu, one, o);
        if (part < 4 && at + (second ? 1 : 0) < live) to[at + (second ? 1 : 0)] = one * factor;
    };

    float P = 1.0f, product = 1.0f;
    for (int t0 = first, b = 0; t0 < last; ++b) {
        const int n = rows_at(t0), t1 = t0 + n;
        float2 next = make_float2(1.0f, 1.0f);
        bool next_direct = false;
        if (t1 < last) {
            const int n1 = rows_at(t1);
            issue(t1, n1, (b + 1) & 1);
            if (!CHANNEL && warp == 0) next = read_facts(t1, n1);
            next_direct = direct_at(t1);
            asm volatile("cp.async.wait_group 1;\n" ::);
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::);
        }
        __syncthreads();
        const float* token = stage + (b & 1) * stage_floats;
        if constexpr (CHANNEL) {
            if (PRODUCTS && slice == 0 && warp == warps - 1) {
                const float* ends = token + A.batch * token_floats;
                for (int i = lane; i < A.d; i += 32) {
                    float p = products[i];
                    if (direct) {
                        for (int j = 0; j < n; ++j) p *= A.keeps[(size_t)(t0 + j) * A.heads * A.d + q_at + i];
                    } else {
                        p *= ends[(i / SCAN_ROWS) * SCAN_PITCH + i % SCAN_ROWS];
                    }
                    products[i] = p;
                }
            }
            if (!idle && direct) {
                for (int j = 0; j < n; ++j, token += token_floats) {
                    const float* keep = A.keeps + (size_t)(t0 + j) * A.heads * A.d + q_at;
#pragma unroll
                    for (int i = 0; i < PAIRS; ++i) {
                        const int row = row0 + 2 * i;
                        const pair f = make_pair(row < A.d ? keep[row] : 0.0f, row + 1 < A.d ? keep[row + 1] : 0.0f);
#pragma unroll
                        for (int c = 0; c < 4; ++c) s[c][i] = mul2(s[c][i], f);
                    }
                    walk(token, 1.0f, 1.0f);
                    to += out_step;
                }
            } else if (!idle) {
                const float* keep = token + A.batch * token_floats + part * SCAN_PITCH;
#pragma unroll 1
                for (int j = 0; j < n; ++j, token += token_floats) {
                    walk(token, 1.0f, 1.0f);
                    to += out_step;
                }
#pragma unroll
                for (int i = 0; i < PAIRS; i += 2) {
                    const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(keep + 2 * i);
#pragma unroll
                    for (int c = 0; c < 4; ++c) s[c][i] = mul2(s[c][i], f.x), s[c][i + 1] = mul2(s[c][i + 1], f.y);
                }
            }
            direct = next_direct;
            t0 = t1;
            __syncthreads();                                 // the stage is copied into again two batches on
            continue;
        }
        const float4* fact = facts[b & 1];
        const float end = fact[n - 1].y;                     // the batch's product of keeps, the same for every thread
        if (MODE == SCAN_LOCAL) product *= end;
        if (P * end < SCAN_LEAST) {
            rescale(P);
            P = 1.0f;
        }
        if (idle) {
        } else if (end < SCAN_LEAST) {
#pragma unroll 1
            for (int j = 0; j < n; ++j, token += token_floats) {
                rescale(fact[j].z);
                walk(token, fact[j].w, 1.0f);
                to += out_step;
            }
        } else {
            const float inverse = 1.0f / P;
#pragma unroll 1
            for (int j = 0; j < n; ++j, token += token_floats) {
                const float2 f = *reinterpret_cast<const float2*>(&fact[j]);
                walk(token, f.x * inverse, f.y * P);
                to += out_step;
            }
        }
        if (end >= SCAN_LEAST) P *= end;
        if (warp == 0 && t1 < last) write_facts(next, (b + 1) & 1);
        t0 = t1;
        __syncthreads();                                     // the stage is copied into again two batches on
    }
    if (MODE == SCAN_LOCAL && !CHANNEL && threadIdx.x == 0 && slice == 0) A.chunk_decay[chunk_at] = product;
    if (PRODUCTS && slice == 0 && warp == warps - 1)
        for (int i = lane; i < A.d; i += 32) A.chunk_decay[chunk_at * A.d + i] = products[i];
    if (MODE == SCAN_LOCAL || (MODE == SCAN_WHOLE && A.write_state)) {
        rescale(P);
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            const float2 x[4] = {split(s[0][i]), split(s[1][i]), split(s[2][i]), split(s[3][i])};
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int row = row0 + 2 * i + u;
                if (row >= A.d) continue;
                const float4 f = u ? make_float4(x[0].y, x[1].y, x[2].y, x[3].y) : make_float4(x[0].x, x[1].x, x[2].x, x[3].x);
                float* to = mine + (size_t)row * A.e + col;
                if (A.vec_state) {
                    if (col < A.e) *reinterpret_cast<float4*>(to) = f;
                } else {
                    if (col < A.e) to[0] = f.x;
                    if (col + 1 < A.e) to[1] = f.y;
                    if (col + 2 < A.e) to[2] = f.z;
                    if (col + 3 < A.e) to[3] = f.w;
                }
                if (is_norm) norm_mine[row] = f.x;
            }
        }
    }
}

// The recurrence for decoded tokens (a token or a few a sequence), where S is read and written once and that is the time: a warp
// takes SCAN_ROWS rows of up to 128 neighbouring columns, four a lane, so that every access is a whole row of them and all of a
// thread's loads are in flight together; the warps' parts of a token's read-out meet in shared memory.  Nothing is staged: k
// and q are the same for a warp's lanes.  At most 16 warps (d up to 256).
// CHANNEL: a warp makes its rows' keeps itself, from the first thin product and its rows of the second (W: their type).
#define STEP_COLUMNS 128
template <bool CHANNEL, typename W>
__global__ void __launch_bounds__(512) linear_step_kernel(const ScanArgs A) {
    __shared__ __align__(16) float parts[2][16][STEP_COLUMNS];
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int seq = blockIdx.x, head = blockIdx.y;
    const int first = A.q_start[seq], last = A.q_start[seq + 1];
    const int slot = A.state_slots[seq];
    if (slot < 0 || last <= first) return;
    const int col = blockIdx.z * STEP_COLUMNS + 4 * lane, row0 = warp * SCAN_ROWS;
    const int norm_col = A.norm_state ? (A.e + 3) / 4 * 4 : -4;
    const bool is_norm = col == norm_col;
    const int live = is_norm ? 1 : min(A.e - col, 4);        // columns of these four that are there
    float* mine = A.state + (long long)slot * A.state_stride + (size_t)head * A.d * A.e + col;
    int step = A.e;                                          // from row to row
    if (is_norm) mine = A.norm_state + (long long)slot * A.state_stride + (size_t)head * A.d, step = 1;
    const bool whole = A.vec_state && !is_norm && live == 4;
    const bool zero = A.positions[first] == 0;
    float4 s[SCAN_ROWS];
#pragma unroll
    for (int i = 0; i < SCAN_ROWS; ++i) {
        s[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        const float* from = mine + (size_t)(row0 + i) * step;
        if (zero || row0 + i >= A.d) continue;
        if (whole) {
            s[i] = *reinterpret_cast<const float4*>(from);
        } else {
            if (live > 0) s[i].x = from[0];
            if (live > 1) s[i].y = from[1];
            if (live > 2) s[i].z = from[2];
            if (live > 3) s[i].w = from[3];
        }
    }
    for (int t = first; t < last; ++t) {
        const size_t row = (size_t)t * A.stride;
        const float *k = A.k + row + head * A.d + row0, *q = A.q + row + head * A.d + row0, *v = A.v + row + head * A.e + col;
        float keep = 1.0f, take = 1.0f;
        if (CHANNEL) {                                       // two lanes a row; lane 2 i ends with the keep of row i
            const int mine_row = row0 + (lane >> 1);
            float z = 0.0f;
            if (mine_row < A.d) {
                const W* up = (const W*)A.up + ((size_t)head * A.d + mine_row) * A.rank;
                const float* low = A.low + row;
                for (int r = lane & 1; r < A.rank; r += 2) z = fmaf(to_float(up[r]), low[r], z);
            }
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            if (mine_row < A.d) keep = channel_keep(z + A.keep_bias[head * A.d + mine_row], A.inverse_tau);
        } else if (A.decay) keep = A.decay[head];
        else keep = A.coef[(size_t)t * A.coef_stride + head], take = A.coef[(size_t)t * A.coef_stride + A.heads + head];
        float4 tv = make_float4(0.0f, 0.0f, 0.0f, 0.0f), y = tv;
        if (is_norm) {
            tv.x = take;                                     // n takes k alone: a column whose value is always 1
        } else {
            if (live > 0) tv.x = take * v[0];
            if (live > 1) tv.y = take * v[1];
            if (live > 2) tv.z = take * v[2];
            if (live > 3) tv.w = take * v[3];
        }
#pragma unroll
        for (int i = 0; i < SCAN_ROWS; i += 4) {
            float4 k4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f), q4 = k4;
            if (A.vec_qk) {
                if (row0 + i < A.d) k4 = *reinterpret_cast<const float4*>(k + i), q4 = *reinterpret_cast<const float4*>(q + i);
            } else {
                if (row0 + i < A.d) k4.x = k[i], q4.x = q[i];
                if (row0 + i + 1 < A.d) k4.y = k[i + 1], q4.y = q[i + 1];
                if (row0 + i + 2 < A.d) k4.z = k[i + 2], q4.z = q[i + 2];
                if (row0 + i + 3 < A.d) k4.w = k[i + 3], q4.w = q[i + 3];
            }
            const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                float4& r = s[i + u];
                const float held = CHANNEL ? __shfl_sync(0xffffffffu, keep, 2 * (i + u)) : keep;
                r.x = fmaf(held, r.x, kk[u] * tv.x), r.y = fmaf(held, r.y, kk[u] * tv.y);
                r.z = fmaf(held, r.z, kk[u] * tv.z), r.w = fmaf(held, r.w, kk[u] * tv.w);
                y.x = fmaf(r.x, qq[u], y.x), y.y = fmaf(r.y, qq[u], y.y), y.z = fmaf(r.z, qq[u], y.z), y.w = fmaf(r.w, qq[u], y.w);
            }
        }
        float (*met)[STEP_COLUMNS] = parts[(t - first) & 1];     // two in turn: one barrier a token is enough
        *reinterpret_cast<float4*>(&met[warp][4 * lane]) = y;
        __syncthreads();
        for (int c = threadIdx.x; c < STEP_COLUMNS; c += blockDim.x) {
            const int at = blockIdx.z * STEP_COLUMNS + c;
            if (at >= A.e && at != norm_col) continue;
            float sum = 0.0f;
            for (int w = 0; w < warps; ++w) sum += met[w][c];
            if (at == norm_col) A.norm_out[(size_t)t * A.heads + head] = sum;
            else A.out[(size_t)t * A.heads * A.e + (size_t)head * A.e + at] = sum;
        }
    }
    if (!A.write_state) return;
#pragma unroll
    for (int i = 0; i < SCAN_ROWS; ++i) {
        float* to = mine + (size_t)(row0 + i) * step;
        if (row0 + i >= A.d) continue;
        if (whole) {
            *reinterpret_cast<float4*>(to) = s[i];
        } else {
            if (live > 0) to[0] = s[i].x;
            if (live > 1) to[1] = s[i].y;
            if (live > 2) to[2] = s[i].z;
            if (live > 3) to[3] = s[i].w;
        }
    }
}

// A thread takes one element (VEC: four neighbouring ones) of a (sequence, head)'s S (and n behind it): chunk c's entry goes from
// the chunk's end state from zero to the state at its start, in[0] = the slot's state (zero at position 0), in[c + 1] =
// product_c in[c] + end_c.  The end states of eight chunks are asked for together.
template <bool VEC, bool CHANNEL>
__global__ void scan_chunk_states_kernel(const ScanArgs A, int elements) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int W = VEC ? 4 : 1, AHEAD = 8;
    const int seq = blockIdx.x, head = blockIdx.y;
    const int first = A.q_start[seq], rows = A.q_start[seq + 1] - first;
    const int slot = A.state_slots[seq];
    if (slot < 0 || rows <= 0) return;
    const int i = (blockIdx.z * blockDim.x + threadIdx.x) * W;
    if (i >= elements) return;
    const int matrix = A.d * A.e;
    const int chunks = CHANNEL ? (first + rows - 1) / A.chunk_len - first / A.chunk_len + 1 : (rows + A.chunk_len - 1) / A.chunk_len;
    const bool fresh = A.positions[first] == 0;
    float* local = A.chunk_state + ((size_t)seq * A.heads + head) * A.max_chunks * A.chunk_floats + i;
    const int products = CHANNEL ? A.d : 1;                  // of a chunk
    const float* product = A.chunk_decay + ((size_t)seq * A.heads + head) * A.max_chunks * products + (CHANNEL ? i / A.e : 0);
    float* slot_at = (i < matrix ? A.state + (size_t)head * matrix + i : A.norm_state + (size_t)head * A.d + (i - matrix)) +
                     (long long)slot * A.state_stride;
    float value[W];
#pragma unroll
    for (int u = 0; u < W; ++u) value[u] = fresh ? 0.0f : slot_at[u];
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float end[AHEAD][W], keep[AHEAD];
#pragma unroll
        for (int c = 0; c < AHEAD; ++c) {
            if (c0 + c >= chunks) continue;
            const float* from = local + (size_t)(c0 + c) * A.chunk_floats;
            keep[c] = product[(size_t)(c0 + c) * products];
            if (VEC) {
                const float4 f = *reinterpret_cast<const float4*>(from);
                end[c][0] = f.x;
                if (VEC) end[c][W > 1 ? 1 : 0] = f.y, end[c][W > 2 ? 2 : 0] = f.z, end[c][W > 3 ? 3 : 0] = f.w;
            } else {
                end[c][0] = from[0];
            }
        }
#pragma unroll
        for (int c = 0; c < AHEAD; ++c) {
            if (c0 + c >= chunks) continue;
            float* to = local + (size_t)(c0 + c) * A.chunk_floats;
            if (VEC) *reinterpret_cast<float4*>(to) = make_float4(value[0], value[W > 1 ? 1 : 0], value[W > 2 ? 2 : 0], value[W > 3 ? 3 : 0]);
            else to[0] = value[0];
#pragma unroll
            for (int u = 0; u < W; ++u) value[u] = fmaf(keep[c], value[u], end[c][u]);
        }
    }
    if (!A.write_state) return;
#pragma unroll
    for (int u = 0; u < W; ++u) slot_at[u] = value[u];
}

}  // namespace

MRS_EXPORT int mrs_rotate_heads(float* rows, int stride, int offset, const float* table, int tokens, int heads, int d, int rot, void* s) {
    if (tokens <= 0 || rot == 0) return 0;
    if (heads <= 0 || d <= 0 || rot < 0 || rot % 2 || rot > d || offset < 0 || offset + heads * d > stride || !table) return MRS_BAD_ARGUMENT;
    const bool vec = rot % 8 == 0 && d % 4 == 0 && stride % 4 == 0 && offset % 4 == 0 && (((uintptr_t)rows | (uintptr_t)table) & 15) == 0;
    const int work = heads * (vec ? rot / 8 : rot / 2);
    const int threads = work >= 256 ? 256 : (work >= 128 ? 128 : 64);
    if (vec)
        MRS_LAUNCH(rotate_heads_kernel<true>, tokens, threads, 0, s, rows, stride, offset, table, tokens, heads, d, rot);
    else
        MRS_LAUNCH(rotate_heads_kernel<false>, tokens, threads, 0, s, rows, stride, offset, table, tokens, heads, d, rot);
    MRS_RETURN_LAUNCH_STATUS();
}

MRS_EXPORT int mrs_narrow_columns(int is_bf16, const float* rows, int stride, int offset, void* out, int tokens, int columns, int live, void* s) {
    if (tokens <= 0 || columns <= 0) return 0;
    if (live < 0 || live > columns || offset < 0 || offset + live > stride) return MRS_BAD_ARGUMENT;
    const long long total = (long long)tokens * columns;
    long long blocks = (total + 255) / 256;
    if (blocks > 8LL * mrs_sm_count()) blocks = 8LL * mrs_sm_count();
    if (is_bf16)
        MRS_LAUNCH(narrow_columns_kernel<bf16>, (unsigned)blocks, 256, 0, s, rows, stride, offset, (bf16*)out, total, columns, live);
    else
        MRS_LAUNCH(narrow_columns_kernel<float>, (unsigned)blocks, 256, 0, s, rows, stride, offset, (float*)out, total, columns, live);
    MRS_RETURN_LAUNCH_STATUS();
}

MRS_EXPORT int mrs_memory_gates(const float* raw, int raw_stride, int i_offset, int f_offset, const float* i_bias, const float* f_bias,
                                float cap, float* m_state, long long state_stride, const int* positions, const int* q_start,
                                const int* state_slots, float* coef, int tokens, int sequences, int heads, int write_state, void* s) {
    if (tokens <= 0 || sequences <= 0) return 0;
    if (heads <= 0 || heads > 65535 || !(cap > 0.0f) || i_offset < 0 || f_offset < 0 || i_offset + heads > raw_stride ||
        f_offset + heads > raw_stride)
        return MRS_BAD_ARGUMENT;
    const int average = tokens / sequences;
    const int threads = average >= 256 ? 512 : (average >= 64 ? 128 : 32);
    MRS_LAUNCH(memory_gates_kernel, dim3(sequences, heads), threads, 0, s, raw, raw_stride, i_offset, f_offset, i_bias, f_bias, cap, m_state,
               state_stride, positions, q_start, state_slots, coef, heads, write_state);
    MRS_RETURN_LAUNCH_STATUS();
}

// Tokens of a batch in shared memory; keeps a channel add one vector a batch.
static int scan_batch(int parts, int cols, bool channel) {
    const int budget = 40 * 1024 / (2 * (int)sizeof(float)) - (channel ? parts * SCAN_PITCH : 0);
    int batch = budget / (2 * parts * SCAN_PITCH + cols);
    if (batch > SCAN_BATCH) batch = SCAN_BATCH;
    if (channel)
        while (batch & (batch - 1)) --batch;                 // batches begin at multiples of their length, and so do chunks
    return batch;
}

// How the recurrence is cut: lanes that share a column group, columns a block, slices of the columns.  Returns the slices.
static int scan_shape(int d, int e, bool normaliser, int* parts_out, int* cols_out) {
    int parts = 1;
    while (parts * SCAN_ROWS < d) parts <<= 1;
    const int per_warp = 4 * (32 / parts);
    int warps = (e + per_warp - 1) / per_warp;
    if (warps > 8) warps = 8;
    *parts_out = parts;
    *cols_out = warps * per_warp;
    const int columns = normaliser ? (e + 3) / 4 * 4 + 4 : e;
    return (columns + *cols_out - 1) / *cols_out;
}

MRS_EXPORT int mrs_linear_scan_slices(int d, int e, int normaliser) {
    int parts, cols;
    if (d <= 0 || d > 512 || e <= 0) return 0;
    return scan_shape(d, e, normaliser != 0, &parts, &cols);
}

// Floats of scratch that a run in chunks needs.  `channel`: keeps a key channel.
MRS_EXPORT long long mrs_linear_scan_scratch_floats(int tokens, int sequences, int heads, int d, int e, int normaliser, int chunk_len,
                                                    int channel) {
    if (chunk_len <= 0) return 0;
    const long long chunks = (tokens + chunk_len - 1) / chunk_len;
    return (long long)sequences * heads * chunks * (((long long)d * e + (normaliser ? d : 0) + 3) / 4 * 4 + (channel ? d : 1));
}

// Rows that a run in chunks of keeps a channel begins its chunks at multiples of (0: sizes that are not built).
MRS_EXPORT int mrs_channel_scan_batch(int d, int e) {
    int parts, cols;
    if (d <= 0 || d > 512 || e <= 0) return 0;
    scan_shape(d, e, false, &parts, &cols);
    return scan_batch(parts, cols, true);
}

// The launches of a recurrence whose inputs and state stand in `A`.
template <bool CHANNEL>
static int scan_run(ScanArgs& A, int tokens, int sequences, int parts, float* scratch, void* s) {
    const int d = A.d, e = A.e, heads = A.heads, chunk_len = A.chunk_len;
    const int threads = A.cols / (4 * (32 / parts)) * 32;
    const int token_floats = 2 * parts * SCAN_PITCH + A.cols;
    const size_t smem = 2 * ((size_t)A.batch * token_floats + (CHANNEL ? parts * SCAN_PITCH : 0)) * sizeof(float);
#define SCAN_LAUNCH(MODE, GRID)                                                                                  \
    switch (parts) {                                                                                             \
        case 1: MRS_LAUNCH((linear_scan_kernel<MODE, 1, CHANNEL>), GRID, threads, smem, s, A); break;             \
        case 2: MRS_LAUNCH((linear_scan_kernel<MODE, 2, CHANNEL>), GRID, threads, smem, s, A); break;             \
        case 4: MRS_LAUNCH((linear_scan_kernel<MODE, 4, CHANNEL>), GRID, threads, smem, s, A); break;             \
        case 8: MRS_LAUNCH((linear_scan_kernel<MODE, 8, CHANNEL>), GRID, threads, smem, s, A); break;             \
        case 16: MRS_LAUNCH((linear_scan_kernel<MODE, 16, CHANNEL>), GRID, threads, smem, s, A); break;           \
        default: MRS_LAUNCH((linear_scan_kernel<MODE, 32, CHANNEL>), GRID, threads, smem, s, A); break;           \
    }
    if (chunk_len == 0) {
        SCAN_LAUNCH(SCAN_WHOLE, dim3(sequences, heads * A.slices));
        MRS_RETURN_LAUNCH_STATUS();
    }
    A.max_chunks = (tokens + chunk_len - 1) / chunk_len;
    if (A.max_chunks > 65535) return MRS_BAD_ARGUMENT;
    const int elements = d * e + (A.norm_state ? d : 0);
    A.chunk_floats = (elements + 3) / 4 * 4;
    A.chunk_state = scratch;
    A.chunk_decay = scratch + (size_t)sequences * heads * A.max_chunks * A.chunk_floats;
    A.vec_state = e % 4 == 0;
    SCAN_LAUNCH(SCAN_LOCAL, dim3(sequences, heads * A.slices, A.max_chunks));
    if (d * e % 4 == 0 && elements % 4 == 0 && A.vec_state)
        MRS_LAUNCH((scan_chunk_states_kernel<true, CHANNEL>), dim3(sequences, heads, (elements / 4 + 127) / 128), 128, 0, s, A, elements);
    else
        MRS_LAUNCH((scan_chunk_states_kernel<false, CHANNEL>), dim3(sequences, heads, (elements + 127) / 128), 128, 0, s, A, elements);
    SCAN_LAUNCH(SCAN_FINAL, dim3(sequences, heads * A.slices, A.max_chunks));
#undef SCAN_LAUNCH
    MRS_RETURN_LAUNCH_STATUS();
}

// q, k, v: pointers to the columns of the first head in float32 rows of `stride` floats.  `chunk_len` 0: in one go.
MRS_EXPORT int mrs_linear_scan(const float* q, const float* k, const float* v, int stride, const float* decay, const float* coef,
                               int coef_stride, float* state, float* norm_state, long long state_stride, const int* positions,
                               const int* q_start, const int* state_slots, float* out, float* norm_out, int tokens, int sequences,
                               int heads, int d, int e, int write_state, int chunk_len, float* scratch, void* s) {
    if (tokens <= 0 || sequences <= 0) return 0;
    if (heads <= 0 || d <= 0 || d > 512 || e <= 0 || chunk_len < 0 || (chunk_len > 0 && !scratch) || (!decay && !coef) ||
        (norm_state && !norm_out) || ((uintptr_t)scratch & 15))
        return MRS_BAD_ARGUMENT;
    ScanArgs A = {};
    int parts, cols;
    const int slices = scan_shape(d, e, norm_state != nullptr, &parts, &cols);
    if ((long long)heads * slices > 65535) return MRS_BAD_ARGUMENT;
    A.q = q, A.k = k, A.v = v, A.stride = stride, A.decay = decay, A.coef = decay ? nullptr : coef, A.coef_stride = coef_stride;
    A.state = state, A.norm_state = norm_state, A.state_stride = state_stride;
    A.positions = positions, A.q_start = q_start, A.state_slots = state_slots, A.out = out, A.norm_out = norm_out;
    A.heads = heads, A.d = d, A.e = e, A.cols = cols, A.slices = slices, A.write_state = write_state, A.chunk_len = chunk_len;
    A.vec_qk = d % 4 == 0 && stride % 4 == 0 && (((uintptr_t)q | (uintptr_t)k) & 15) == 0;
    A.vec_v = e % 4 == 0 && stride % 4 == 0 && ((uintptr_t)v & 15) == 0;
    A.vec_out = e % 4 == 0 && ((uintptr_t)out & 15) == 0;
    A.vec_state = e % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    if (chunk_len == 0 && d <= 256 && tokens < 4LL * sequences) {
        const int columns = norm_state ? (e + 3) / 4 * 4 + 4 : e;
        MRS_LAUNCH((linear_step_kernel<false, float>), dim3(sequences, heads, (columns + STEP_COLUMNS - 1) / STEP_COLUMNS),
                   (d + SCAN_ROWS - 1) / SCAN_ROWS * 32, 0, s, A);
        MRS_RETURN_LAUNCH_STATUS();
    }
    int batch = scan_batch(parts, cols, false);
    if (tokens < SCAN_BATCH * sequences && batch > (tokens + sequences - 1) / sequences) batch = (tokens + sequences - 1) / sequences;
    if (batch < 1) return MRS_BAD_ARGUMENT;
    A.batch = batch;
    return scan_run<false>(A, tokens, sequences, parts, scratch, s);
}

// The recurrence with keeps a key channel, made here: sigmoid(up low + bias)^(inverse_tau), `low` pointing to `rank` columns of the
// rows that hold q, k and v, `up` [heads * d, rank] in float32 or bfloat16, `bias` [heads * d].  In portions q and k are changed in
// place; `keeps` [tokens, heads * d] and `direct` [tokens, heads] are scratch.  A run in chunks wants chunks of a multiple of
// mrs_channel_scan_batch rows.
MRS_EXPORT int mrs_channel_scan(float* q, float* k, const float* v, int stride, const float* low, int rank, const void* up, int up_is_bf16,
                                const float* bias, float inverse_tau, float* keeps, int* direct, float* state, long long state_stride,
                                const int* positions, const int* seq_of_token, const int* q_start, const int* state_slots, float* out,
                                int tokens, int sequences, int heads, int d, int e, int write_state, int chunk_len, float* scratch, void* s) {
    if (tokens <= 0 || sequences <= 0) return 0;
    if (heads <= 0 || d <= 0 || d > 512 || e <= 0 || rank <= 0 || rank > 1024 || chunk_len < 0 || (chunk_len > 0 && !scratch) || !up || !bias ||
        !keeps || !direct || !(inverse_tau > 0.0f) || ((uintptr_t)scratch & 15))
        return MRS_BAD_ARGUMENT;
    ScanArgs A = {};
    int parts, cols;
    const int slices = scan_shape(d, e, false, &parts, &cols);
    if ((long long)heads * slices > 65535) return MRS_BAD_ARGUMENT;
    A.q = q, A.k = k, A.v = v, A.stride = stride, A.low = low, A.rank = rank, A.up = up, A.keep_bias = bias, A.inverse_tau = inverse_tau;
    A.keeps = keeps, A.direct = direct, A.state = state, A.state_stride = state_stride;
    A.positions = positions, A.q_start = q_start, A.state_slots = state_slots, A.out = out;
    A.heads = heads, A.d = d, A.e = e, A.cols = cols, A.slices = slices, A.write_state = write_state, A.chunk_len = chunk_len;
    A.vec_qk = d % 4 == 0 && stride % 4 == 0 && (((uintptr_t)q | (uintptr_t)k) & 15) == 0;
    A.vec_v = e % 4 == 0 && stride % 4 == 0 && ((uintptr_t)v & 15) == 0;
    A.vec_out = e % 4 == 0 && ((uintptr_t)out & 15) == 0;
    A.vec_state = e % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    A.vec_keeps = d % 4 == 0 && ((uintptr_t)keeps & 15) == 0;
    if (chunk_len == 0 && d <= 256 && tokens < 4LL * sequences) {
        const dim3 grid(sequences, heads, (e + STEP_COLUMNS - 1) / STEP_COLUMNS);
        const int threads = (d + SCAN_ROWS - 1) / SCAN_ROWS * 32;
        if (up_is_bf16) MRS_LAUNCH((linear_step_kernel<true, bf16>), grid, threads, 0, s, A);
        else MRS_LAUNCH((linear_step_kernel<true, float>), grid, threads, 0, s, A);
        MRS_RETURN_LAUNCH_STATUS();
    }
    A.batch = scan_batch(parts, cols, true);
    if (A.batch < 1 || chunk_len % A.batch) return MRS_BAD_ARGUMENT;
    int heads_a_block = 256 / d;
    if (heads_a_block < 1) heads_a_block = 1;
    if (heads_a_block > 32) heads_a_block = 32;
    if (heads_a_block > heads) heads_a_block = heads;
    const dim3 grid((tokens + A.batch - 1) / A.batch, (heads + heads_a_block - 1) / heads_a_block);
    const int threads = (heads_a_block * d + 31) / 32 * 32;
    const size_t smem = (size_t)SCAN_BATCH * rank * sizeof(float);
    if (up_is_bf16) MRS_LAUNCH(channel_fold_kernel<bf16>, grid, threads, smem, s, A, q, k, seq_of_token, tokens, heads_a_block);
    else MRS_LAUNCH(channel_fold_kernel<float>, grid, threads, smem, s, A, q, k, seq_of_token, tokens, heads_a_block);
    return scan_run<true>(A, tokens, sequences, parts, scratch, s);
}
