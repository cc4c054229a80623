// The gated delta rule: a recurrence whose state is a matrix S [d, e] per (request, head) that forgets by a scalar a
// token and then corrects what it holds under the token's key towards the token's value:
//
//     S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
// with q_t, k_t [d] (shared by the query heads of a group) made unit vectors, x / sqrt(sum x^2 + unit_eps), q also times
// a constant; beta_t = sigmoid(b_t); g_t = exp(-exp(A_log_h) softplus(a_t + dt_bias_h)), one a head, or one a head and key
// channel (g_t [d] then acts on the rows of S).  Afterwards every head's o_t is divided by its root mean square, multiplied
// by a weight and by silu or sigmoid of a gate.
//
// Everything here is float32: unit norms, step sizes, decays, the state and the read-out.  S lives in the request's
// state slot between steps [slots, heads, d, e]; where a sequence starts at position 0 its state counts as zero, whatever
// the slot held (slots are used again).  State slot -1: a padding sequence, nothing is read or written.  The step's
// facts come from device arrays only, so a step can be recorded.
//
//   delta_prepare     per token: q and k of every group to unit length in place; beta and g of every head (or beta, and in
//                     place the g of every head and channel)
//   delta_scan        the recurrence token by token; one block a (sequence, head, slice of S's columns), the tokens'
//                     inputs staged through shared memory ahead of their use
//   head_norm_gate    o / rms(o) * weight * act(gate) per (token, head), o first divided by a normaliser where there is one
#include "common.cuh"
#include "pairs.cuh"

namespace {

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// qkv [tokens, 2 * groups * d + heads * e] float32: q of every group, k of every group, v of every head.
// raw [tokens, raw_stride] float32: at column b_offset one b a head, at a_offset one a a head.
// coef [tokens, 2 * heads]: beta, then g.  With `channels` (rows of `channels_stride` floats, heads * d columns of raw decays,
// dt_bias one a column) the decays are made there in place and coef is [tokens, heads]: beta.
__global__ void delta_prepare_kernel(float* __restrict__ qkv, int qkv_width, const float* __restrict__ raw, int raw_stride,
                                     int b_offset, int a_offset, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                     float* __restrict__ coef, float* __restrict__ channels, int channels_stride, int groups, int d,
                                     int heads, float unit_eps, float q_factor) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), warps = gridDim.y * (blockDim.x >> 5);
    float* row = qkv + t * qkv_width;
    for (int unit = warp; unit < 2 * groups; unit += warps) {          // units 0 .. groups - 1: q; the rest: k
        float* x = row + (size_t)unit * d;
        float sum = 0.0f;
        for (int i = lane; i < d; i += 32) sum += x[i] * x[i];
        const float factor = (unit < groups ? q_factor : 1.0f) / sqrtf(warp_sum(sum) + unit_eps);
        for (int i = lane; i < d; i += 32) x[i] *= factor;
    }
    const float* r = raw + t * raw_stride;
    if (channels) {
        if (blockIdx.y == 0)
            for (int h = threadIdx.x; h < heads; h += blockDim.x) coef[t * heads + h] = 1.0f / (1.0f + expf(-r[b_offset + h]));
        float* z = channels + t * channels_stride;
        for (int h = warp; h < heads; h += warps) {
            const float rate = -expf(a_log[h]);
            for (int i = h * d + lane; i < (h + 1) * d; i += 32) z[i] = expf(rate * softplus_f(z[i] + dt_bias[i]));
        }
        return;
    }
    if (blockIdx.y != 0) return;
    for (int h = threadIdx.x; h < heads; h += blockDim.x) {
        coef[t * 2 * heads + h] = 1.0f / (1.0f + expf(-r[b_offset + h]));
        coef[t * 2 * heads + heads + h] = expf(-expf(a_log[h]) * softplus_f(r[a_offset + h] + dt_bias[h]));
    }
}

__device__ __forceinline__ uint32_t shared_address(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void copy_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(shared_address(dst)), "l"(src));
}
__device__ __forceinline__ void copy_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(shared_address(dst)), "l"(src));
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

// Thread (column c of the block's slice, part p): rows p * PER .. p * PER + PER - 1 of column c of S in registers, two to a
// register pair (PER is 16 or 8, the launcher's choice); the PARTS lanes of one column lie in one warp, so that the two sums
// over d are log2(PARTS) shuffles.  The tokens' inputs (k and
// q of the head's group, the slice of v, beta and g; CHANNEL: also the head's d decays) come in batches of `batch_tokens` through two stages of shared memory:
// the next batch is copied while this one is computed, and the threads of a block share what they read.  A token in shared
// memory: k [PARTS * PITCH] | q [PARTS * PITCH] (| decays [PARTS * PITCH]) | v [cols rounded up to 4] | beta, g, 0, 0, with PITCH = PER + 4, so that
// the 16-byte reads of the parts fall on different banks; the rows beyond d stay zero.
//
// One warp a scheduler is all that a single sequence offers, so every instruction's latency shows.  What a thread copies is
// therefore the same in every batch and worked out once, ahead of the loop (`Copies`); and the chain from token to token is only: the sum over S's old rows times k (CHANNEL: times k
// already multiplied by the decays), the shuffles, u, one fused multiply-add a row.  The decay is applied to S beside the
// shuffles, and a token's read-out is summed over its lanes by the next token's shuffles.
template <int N>
struct Copies {
    int src[N], dst[N], token[N];      // offsets in floats from the batch's first row and from the stage; a huge token: none
};

// What a thread needs of one token.
template <int PER, bool CHANNEL>
struct Token {
    pair k[PER / 2], q[PER / 2], fade[CHANNEL ? PER / 2 : 1], faded[CHANNEL ? PER / 2 : 1];      // faded: k times the decays
    float v, beta, decay;

    __device__ __forceinline__ void read(const float* token, int rows, int tail_at, int cols_pad, int col_in_slice) {
#pragma unroll
        for (int i = 0; i < PER / 2; i += 2) {
            const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(token + 2 * i);
            const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(token + rows + 2 * i);
            k[i] = kk.x, k[i + 1] = kk.y, q[i] = qq.x, q[i + 1] = qq.y;
            if (CHANNEL) {
                const ulonglong2 ff = *reinterpret_cast<const ulonglong2*>(token + 2 * rows + 2 * i);
                fade[i] = ff.x, fade[i + 1] = ff.y;
                faded[i] = mul2(kk.x, ff.x), faded[i + 1] = mul2(kk.y, ff.y);
            }
        }
        const float* tail = token + tail_at;
        v = (tail - cols_pad)[col_in_slice], beta = tail[0], decay = CHANNEL ? 1.0f : tail[1];
    }
};

template <int PER, int PARTS, bool CHANNEL>
__global__ void __launch_bounds__(128) delta_scan_kernel(const float* __restrict__ qkv, int qkv_width, const float* __restrict__ coef,
                                  const float* __restrict__ channels, int channels_stride,
                                  float* __restrict__ state, long long state_stride, const int* __restrict__ positions,
                                  const int* __restrict__ q_start, const int* __restrict__ state_slots, float* __restrict__ out,
                                  int heads, int groups, int d, int e, int cols, int batch_tokens, int wide_copies,
                                  int write_state) {
    extern __shared__ __align__(16) float stage[];
    constexpr int PITCH = PER + 4, ROWS = PARTS * PITCH, VECTORS = CHANNEL ? 3 : 2;
    constexpr int FACTS = CHANNEL ? 1 : 2;                 // beta, and the decay of the head
    constexpr int WIDE = 8, NARROW = 3;                    // copies a thread and batch that are worked out ahead
    pdl_launch_dependents();
    const int cols_pad = (cols + 3) & ~3;
    const int token_floats = VECTORS * ROWS + cols_pad + 4, stage_floats = batch_tokens * token_floats;
    for (int i = threadIdx.x; i < 2 * stage_floats; i += blockDim.x) stage[i] = 0.0f;
    __syncthreads();
    pdl_wait();
    const int seq = blockIdx.x, head = blockIdx.y;
    const int first = q_start[seq], last = q_start[seq + 1];
    const int slot = state_slots[seq];
    if (slot < 0 || last <= first) return;
    // a warp's GROUPS columns lie side by side in its lanes: a 16-byte read by half a warp then has few distinct addresses
    constexpr int GROUPS = 32 / PARTS;
    const int lane = threadIdx.x & 31, part = lane / GROUPS, col_in_slice = (threadIdx.x >> 5) * GROUPS + lane % GROUPS;
    const int col = blockIdx.z * cols + col_in_slice;
    const bool live = col < e;                       // a slice may overhang the head; its threads still take part in the shuffles
    const int c = live ? col : 0;
    const int group = head / (heads / groups);
    const int row0 = part * PER;
    float* mine = state + (long long)slot * state_stride + ((size_t)head * d) * e + c;
    pair s[PER / 2];                                 // the rows two by two
    const bool fresh = positions[first] == 0;
#pragma unroll
    for (int i = 0; i < PER; i += 2)
        s[i / 2] = make_pair((!fresh && live && row0 + i < d) ? mine[(size_t)(row0 + i) * e] : 0.0f,
                             (!fresh && live && row0 + i + 1 < d) ? mine[(size_t)(row0 + i + 1) * e] : 0.0f);

    const int q_at = group * d, k_at = (groups + group) * d, v_at = 2 * groups * d + head * e + (int)blockIdx.z * cols;
    const int live_cols = min(cols, e - (int)blockIdx.z * cols);
    // copy number i of a batch's keys and queries (and decays): token j, k, q or decays, elements el .. of the vector
    const int width = wide_copies ? d >> 2 : d, vector_copies = batch_tokens * VECTORS * width;
    auto vector_copy = [&](int i, int& src, int& dst) {
        const int j = i / (VECTORS * width), r = i % (VECTORS * width), which = r / width, el = (r % width) * (wide_copies ? 4 : 1);
        if (CHANNEL && which == 2) src = -1 - (j * channels_stride + head * d + el);          // below zero: from the decays
        else src = j * qkv_width + (which ? q_at : k_at) + el;
        dst = j * token_floats + which * ROWS + (el / PER) * PITCH + el % PER;
        return j;
    };
    // copy number i of a batch's values and coefficients: token j, a column of v, beta or g
    const int scalar_copies = batch_tokens * (live_cols + FACTS);
    auto scalar_copy = [&](int i, long long& src, int& dst) {
        const int j = i / (live_cols + FACTS), r = i % (live_cols + FACTS);
        if (r < live_cols) {
            src = (long long)j * qkv_width + v_at + r;
            dst = j * token_floats + VECTORS * ROWS + r;
        } else {
            src = -1 - ((long long)j * FACTS * heads + (r == live_cols ? head : heads + head));      // below zero: from coef
            dst = j * token_floats + VECTORS * ROWS + cols_pad + (r - live_cols);
        }
        return j;
    };
    Copies<WIDE> wide;
    Copies<NARROW> narrow;
    long long narrow_src[NARROW];
    const int longest = min(batch_tokens, last - first);       // a decoded token alone needs the first token's copies only
#pragma unroll
    for (int i = 0; i < WIDE; ++i) {
        const int at = threadIdx.x + i * blockDim.x;
        wide.token[i] = at < longest * VECTORS * width ? vector_copy(at, wide.src[i], wide.dst[i]) : (1 << 30);
    }
#pragma unroll
    for (int i = 0; i < NARROW; ++i) {
        const int at = threadIdx.x + i * blockDim.x;
        narrow.token[i] = at < longest * (live_cols + FACTS) ? scalar_copy(at, narrow_src[i], narrow.dst[i]) : (1 << 30);
    }
    auto issue = [&](int t0, int n, int buffer) {
        float* base = stage + buffer * stage_floats;
        const float* rows = qkv + (size_t)t0 * qkv_width;
        const float* facts = coef + (size_t)t0 * FACTS * heads;
        const float* fades = CHANNEL ? channels + (size_t)t0 * channels_stride : nullptr;
#pragma unroll
        for (int i = 0; i < WIDE; ++i)
            if (wide.token[i] < n) {
                const float* from = CHANNEL && wide.src[i] < 0 ? fades + (-1 - wide.src[i]) : rows + wide.src[i];
                if (wide_copies) copy_async16(base + wide.dst[i], from);
                else copy_async4(base + wide.dst[i], from);
            }
        for (int at = threadIdx.x + WIDE * blockDim.x; at < vector_copies; at += blockDim.x) {      // sizes beyond the usual
            int src, dst;
            if (vector_copy(at, src, dst) < n) {
                const float* from = CHANNEL && src < 0 ? fades + (-1 - src) : rows + src;
                if (wide_copies) copy_async16(base + dst, from);
                else copy_async4(base + dst, from);
            }
        }
#pragma unroll
        for (int i = 0; i < NARROW; ++i)
            if (narrow.token[i] < n) copy_async4(base + narrow.dst[i], narrow_src[i] >= 0 ? rows + narrow_src[i] : facts + (-1 - narrow_src[i]));
        for (int at = threadIdx.x + NARROW * blockDim.x; at < scalar_copies; at += blockDim.x) {
            long long src;
            int dst;
            if (scalar_copy(at, src, dst) < n) copy_async4(base + dst, src >= 0 ? rows + src : facts + (-1 - src));
        }
        copy_async_commit();
    };
    const int batches = (last - first + batch_tokens - 1) / batch_tokens;
    const int token_tail = VECTORS * ROWS + cols_pad;
    float* out_at = out + (size_t)first * heads * e + (size_t)head * e + c;
    const size_t out_step = (size_t)heads * e;
    const bool writes = live && part == 0;
    float y = 0.0f;                                       // this lane's part of the last token's read-out
    bool pending = false;
    issue(first, min(batch_tokens, last - first), 0);
    for (int b = 0; b < batches; ++b) {
        const int t0 = first + b * batch_tokens, n = min(batch_tokens, last - t0);
        if (b + 1 < batches) {
            issue(t0 + batch_tokens, min(batch_tokens, last - t0 - batch_tokens), (b + 1) & 1);
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        const float* token = stage + (b & 1) * stage_floats + part * PITCH;
#pragma unroll 1
        for (int j = 0; j < n; ++j, token += token_floats) {
            Token<PER, CHANNEL> now;
            now.read(token, ROWS, token_tail - part * PITCH, cols_pad, col_in_slice);
            pair r2[2] = {0ull, 0ull};
#pragma unroll
            for (int i = 0; i < PER / 2; ++i) r2[i & 1] = fma2(s[i], CHANNEL ? now.faded[CHANNEL ? i : 0] : now.k[i], r2[i & 1]);
            float r = both(r2[0]) + both(r2[1]);
#pragma unroll
            for (int o = GROUPS; o < 32; o <<= 1) {                   // this token's sum and the one before's read-out side by side
                const float other_r = __shfl_xor_sync(0xffffffffu, r, o), other_y = __shfl_xor_sync(0xffffffffu, y, o);
                r += other_r, y += other_y;
            }
            if (writes && pending) *out_at = y, out_at += out_step;
            pending = true;
            const pair decays = make_pair(now.decay, now.decay);
#pragma unroll
            for (int i = 0; i < PER / 2; ++i) s[i] = mul2(s[i], CHANNEL ? now.fade[CHANNEL ? i : 0] : decays);      // off the chain
            const float u = now.beta * (now.v - (CHANNEL ? r : now.decay * r));
            const pair uu = make_pair(u, u);
            pair y2[2] = {0ull, 0ull};
#pragma unroll
            for (int i = 0; i < PER / 2; ++i) {
                s[i] = fma2(now.k[i], uu, s[i]);
                y2[i & 1] = fma2(s[i], now.q[i], y2[i & 1]);
            }
            y = both(y2[0]) + both(y2[1]);
        }
        __syncthreads();                                  // the stage is copied into again two batches on
    }
#pragma unroll
    for (int o = GROUPS; o < 32; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (writes) *out_at = y;                              // the last token's
    if (write_state && live) {
#pragma unroll
        for (int i = 0; i < PER; i += 2) {
            const float2 x = split(s[i / 2]);
            if (row0 + i < d) mine[(size_t)(row0 + i) * e] = x.x;
            if (row0 + i + 1 < d) mine[(size_t)(row0 + i + 1) * e] = x.y;
        }
    }
}

// One warp a (token, head): x = o * factor (/ (max(|c * factor|, floor) + floor_eps) where there is a normaliser c), then
// out = x / sqrt(mean(x^2) + eps) * weight * act(gate), act = silu or (SIGMOID) the sigmoid.  o [tokens, heads * e] float32;
// gate a column range of wider float32 rows; weight [e] shared by the heads (weight_stride 0), [heads, e] (weight_stride e) or
// null; c [tokens, heads], floor [tokens, floor_stride] from its first column on.
struct HeadNorm {
    const float *o, *gate, *weight, *c, *floor;
    int gate_stride, weight_stride, floor_stride, tokens, heads, e;
    float eps, factor, floor_eps;
};

template <bool SIGMOID> __device__ __forceinline__ float gate_of(float g) {
    const float s = 1.0f / (1.0f + expf(-g));
    return SIGMOID ? s : g * s;
}

__device__ __forceinline__ float head_factor(const HeadNorm& A, size_t t, int h) {
    if (!A.c) return A.factor;
    return A.factor / (fmaxf(fabsf(A.c[t * A.heads + h] * A.factor), A.floor[t * A.floor_stride + h]) + A.floor_eps);
}

template <typename T, bool SIGMOID>
__global__ void head_norm_gate_kernel(const HeadNorm A, T* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, e = A.e;
    const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= (long long)A.tokens * A.heads) return;
    const size_t t = (size_t)(unit / A.heads);
    const int h = (int)(unit % A.heads);
    const float* x = A.o + t * A.heads * e + (size_t)h * e;
    const float* g = A.gate + t * A.gate_stride + (size_t)h * e;
    const float* w = A.weight ? A.weight + (size_t)h * A.weight_stride : nullptr;
    const float factor = head_factor(A, t, h);
    float sum = 0.0f;
    for (int i = lane; i < e; i += 32) sum += (x[i] * factor) * (x[i] * factor);
    const float scale = 1.0f / sqrtf(warp_sum(sum) / (float)e + A.eps);
    T* dst = out + t * A.heads * e + (size_t)h * e;
    for (int i = lane; i < e; i += 32) {
        const float y = x[i] * factor * scale;
        dst[i] = from_float<T>((w ? y * w[i] : y) * gate_of<SIGMOID>(g[i]));
    }
}

template <typename T> __device__ __forceinline__ void put_four(T* p, float4 v);
template <> __device__ __forceinline__ void put_four<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void put_four<bf16>(bf16* p, float4 v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&lo);
    raw.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}

// Heads of a multiple of four elements in rows on 16-byte boundaries, at most 128 * NV: four elements a lane and access, all of a
// head's loads in flight together.  LANES lanes a head (32, or 16 for heads of up to 64 elements).
template <typename T, bool SIGMOID, int NV, int LANES>
__global__ void head_norm_gate_vec_kernel(const HeadNorm A, T* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x % LANES, e = A.e;
    const long long units = (long long)A.tokens * A.heads;
    long long unit = (long long)blockIdx.x * (blockDim.x / LANES) + threadIdx.x / LANES;
    const bool live = unit < units;
    if (!live) unit = units - 1;                             // its lanes still take part in the shuffles
    const size_t t = (size_t)(unit / A.heads);
    const int h = (int)(unit % A.heads);
    const float* x = A.o + t * A.heads * e + (size_t)h * e;
    const float* g = A.gate + t * A.gate_stride + (size_t)h * e;
    float4 v[NV], gates[NV];
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = 4 * (lane + j * LANES);
        v[j] = gates[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (i < e) v[j] = *reinterpret_cast<const float4*>(x + i), gates[j] = *reinterpret_cast<const float4*>(g + i);
    }
    const float factor = head_factor(A, t, h);
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        v[j].x *= factor, v[j].y *= factor, v[j].z *= factor, v[j].w *= factor;
        sum += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    const float scale = 1.0f / sqrtf(sum / (float)e + A.eps);
    if (!live) return;
    T* dst = out + t * A.heads * e + (size_t)h * e;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = 4 * (lane + j * LANES);
        if (i >= e) continue;
        float4 w = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
        if (A.weight) w = *reinterpret_cast<const float4*>(A.weight + (size_t)h * A.weight_stride + i);
        put_four<T>(dst + i, make_float4(v[j].x * scale * w.x * gate_of<SIGMOID>(gates[j].x), v[j].y * scale * w.y * gate_of<SIGMOID>(gates[j].y),
                                         v[j].z * scale * w.z * gate_of<SIGMOID>(gates[j].z), v[j].w * scale * w.w * gate_of<SIGMOID>(gates[j].w)));
    }
}

}  // namespace

MRS_EXPORT int mrs_delta_prepare(float* qkv, const float* raw, int raw_stride, int b_offset, int a_offset, const float* a_log,
                                 const float* dt_bias, float* coef, float* channels, int channels_stride, int tokens, int groups, int d,
                                 int heads, int e, float unit_eps, float q_factor, void* stream) {
    if (tokens <= 0) return 0;
    if (groups <= 0 || d <= 0 || heads <= 0 || e <= 0 || heads % groups) return MRS_BAD_ARGUMENT;
    const int units = 2 * groups;
    const int threads = units >= 8 || channels ? 256 : (units >= 4 ? 128 : 64);
    const int across = channels && tokens < mrs_sm_count() ? 4 : 1;      // few tokens: their heads' decays over several blocks
    MRS_LAUNCH(delta_prepare_kernel, dim3(tokens, across), threads, 0, stream, qkv, 2 * groups * d + heads * e, raw, raw_stride, b_offset, a_offset,
               a_log, dt_bias, coef, channels, channels_stride, groups, d, heads, unit_eps, q_factor);
    MRS_RETURN_LAUNCH_STATUS();
}

// state [slots, heads, d, e] float32 with `state_stride` floats from slot to slot; out [tokens, heads * e] float32.
// `channels`: the decays of every head and channel, rows of `channels_stride` floats (null: one a head, in coef).
MRS_EXPORT int mrs_delta_scan(const float* qkv, const float* coef, const float* channels, int channels_stride, float* state, long long state_stride, const int* positions,
                              const int* q_start, const int* state_slots, float* out, int tokens, int sequences, int heads,
                              int groups, int d, int e, int write_state, void* stream) {
    if (tokens <= 0 || sequences <= 0) return 0;
    if (groups <= 0 || d <= 0 || d > 512 || heads <= 0 || e <= 0 || heads % groups || heads > 65535) return MRS_BAD_ARGUMENT;
    const long long pairs = (long long)sequences * heads;
    int per, parts, cols, slices;
    auto plan = [&](int rows) {
        per = rows;
        parts = 1;
        while (parts * per < d) parts <<= 1;             // lanes a column: a power of two, at most 32
        // columns a block: four warps' worth of threads (they share the tokens' keys and queries in shared memory), fewer
        // while the blocks would leave half the multiprocessors idle, at least a warp's worth of threads
        cols = 128 / parts;
        while (cols > e && cols * parts > 32) cols >>= 1;
        while (cols * parts > 32 && pairs * ((e + cols - 1) / cols) * 2 < mrs_sm_count()) cols >>= 1;
        slices = (e + cols - 1) / cols;
    };
    // rows of a column a thread: 16; 8 where long portions come as more blocks than multiprocessors, so that more of them
    // are resident side by side (measured: from 1.1 to 1.3 times as fast there, slower for short portions and few blocks), and
    // for all long portions with a decay a channel (535 against 624 us for 2,048 tokens of 16 heads)
    plan(16);
    if (d <= 256 && tokens >= 256LL * sequences && (channels || pairs * slices > mrs_sm_count())) plan(8);
    if (slices > 65535) return MRS_BAD_ARGUMENT;
    const int qkv_width = 2 * groups * d + heads * e;
    const int token_floats = (channels ? 3 : 2) * parts * (per + 4) + ((cols + 3) & ~3) + 4;
    int batch_tokens = (48 * 1024) / (2 * token_floats * (int)sizeof(float));
    if (batch_tokens > 8) batch_tokens = 8;
    if (batch_tokens < 1) return MRS_BAD_ARGUMENT;
    const int wide_copies = d % 4 == 0 && qkv_width % 4 == 0 && ((uintptr_t)qkv & 15) == 0 &&
                            (!channels || (channels_stride % 4 == 0 && ((uintptr_t)channels & 15) == 0));
    const dim3 grid(sequences, heads, slices);
    const size_t shared = 2 * (size_t)batch_tokens * token_floats * sizeof(float);
#define MRS_DELTA_SCAN(PER, PARTS, CHANNEL)                                                                                          \
    MRS_LAUNCH((delta_scan_kernel<PER, PARTS, CHANNEL>), grid, cols * PARTS, shared, stream, qkv, qkv_width, coef, channels,         \
               channels_stride, state, state_stride, positions, q_start, state_slots, out, heads, groups, d, e, cols, batch_tokens,  \
               wide_copies, write_state)
#define MRS_DELTA_SCAN_ROWS(PER, CHANNEL)                                                                                            \
    switch (parts) {                                                                                                                 \
        case 1: MRS_DELTA_SCAN(PER, 1, CHANNEL); break;                                                                              \
        case 2: MRS_DELTA_SCAN(PER, 2, CHANNEL); break;                                                                              \
        case 4: MRS_DELTA_SCAN(PER, 4, CHANNEL); break;                                                                              \
        case 8: MRS_DELTA_SCAN(PER, 8, CHANNEL); break;                                                                              \
        case 16: MRS_DELTA_SCAN(PER, 16, CHANNEL); break;                                                                            \
        default: MRS_DELTA_SCAN(PER, 32, CHANNEL); break;                                                                            \
    }
    if (channels) {
        if (per == 16) { MRS_DELTA_SCAN_ROWS(16, true) } else { MRS_DELTA_SCAN_ROWS(8, true) }
    } else {
        if (per == 16) { MRS_DELTA_SCAN_ROWS(16, false) } else { MRS_DELTA_SCAN_ROWS(8, false) }
    }
#undef MRS_DELTA_SCAN_ROWS
#undef MRS_DELTA_SCAN
    MRS_RETURN_LAUNCH_STATUS();
}

MRS_EXPORT int mrs_head_norm_gate(int is_bf16, const float* o, const float* gate, int gate_stride, int sigmoid, const float* weight,
                                  int weight_stride, float eps, float factor, const float* c, const float* floor, int floor_stride,
                                  float floor_eps, void* out, int tokens, int heads, int e, void* stream) {
    if (tokens <= 0) return 0;
    if (heads <= 0 || e <= 0 || (c && !floor)) return MRS_BAD_ARGUMENT;
    HeadNorm A = {o, gate, weight, c, floor, gate_stride, weight_stride, floor_stride, tokens, heads, e, eps, factor, floor_eps};
    const long long units = (long long)tokens * heads;
    const bool vec = e % 4 == 0 && e <= 512 && gate_stride % 4 == 0 && (((uintptr_t)o | (uintptr_t)gate | (uintptr_t)weight | (uintptr_t)out) & 15) == 0;
    const int per_block = vec && e <= 64 ? 8 : 4;
    const unsigned blocks = (unsigned)((units + per_block - 1) / per_block);
#define MRS_HEAD_NORM(T, SIGMOID)                                                                                                \
    do {                                                                                                                         \
        if (!vec) MRS_LAUNCH((head_norm_gate_kernel<T, SIGMOID>), blocks, 128, 0, stream, A, (T*)out);                            \
        else if (e <= 64) MRS_LAUNCH((head_norm_gate_vec_kernel<T, SIGMOID, 1, 16>), blocks, 128, 0, stream, A, (T*)out);         \
        else if (e <= 128) MRS_LAUNCH((head_norm_gate_vec_kernel<T, SIGMOID, 1, 32>), blocks, 128, 0, stream, A, (T*)out);        \
        else if (e <= 256) MRS_LAUNCH((head_norm_gate_vec_kernel<T, SIGMOID, 2, 32>), blocks, 128, 0, stream, A, (T*)out);        \
        else MRS_LAUNCH((head_norm_gate_vec_kernel<T, SIGMOID, 4, 32>), blocks, 128, 0, stream, A, (T*)out);                      \
    } while (0)
    if (is_bf16) {
        if (sigmoid) MRS_HEAD_NORM(bf16, true); else MRS_HEAD_NORM(bf16, false);
    } else {
        if (sigmoid) MRS_HEAD_NORM(float, true); else MRS_HEAD_NORM(float, false);
    }
#undef MRS_HEAD_NORM
    MRS_RETURN_LAUNCH_STATUS();
}
