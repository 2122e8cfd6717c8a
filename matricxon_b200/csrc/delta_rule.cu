// The gated delta rule: per value head a matrix state S [dim][vdim] that forgets, corrects itself and is read.
//
//   S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q      (g: one number per head, or one per row of S)
//
// q, k and v arrive as projections and pass a causal convolution over time per channel and silu; q and k are made unit
// vectors per head. Everything here is float: the projections' float accumulators, the convolution's kept inputs, unit
// norms, steps, decays, state and read-outs.
//
// A request's state vector holds the convolutions' latest taps - 1 inputs [taps - 1][C] (C = 2 q/k heads x dim + heads x
// vdim channels, in the projection's order q | k | v) and, from `state_offset`, S transposed: [heads][vdim][dim], so that a
// value column's dim entries lie side by side. Head sizes are padded to multiples of four by the caller (zero weights make
// zero entries, which change nothing); a mean over a head's values divides by its true width.
//
// mx_delta_prepare: projection rows -> qkv [tokens][C] (unit q times q_scale | unit k | v), beta = sigmoid(b) and, where the
//   decay is one number per head, g = exp(rate_h softplus(a + dt_bias_h)) with rate = -exp(A_log). A warp owns a head (or
//   128 value channels) and walks neighbouring tokens with the convolution's window in registers. The memory of sequences
//   that bring one token is moved on here, that of the others by mx_conv_state_update afterwards.
// mx_delta_decay: g for every head and key channel from a low-rank row: exp(rate_h softplus(A2 low + dt_bias)); a thread per
//   channel keeps its row of A2 in registers for sixteen tokens.
// mx_delta_scan: every sequence's tokens in order, eight at a time. Within a group of eight the writes u solve a triangular
//   system whose coefficients do not depend on the state: u = T (v - S^T k'), o = S^T q' + P u, S <- G S + k'' u^T with k', q'
//   decayed from the group's start, k'' to its end, G over the whole group, T and P 8 x 8. A first kernel forms them for
//   all groups in parallel (decays enter as products of numbers up to one, nothing is divided); the second walks the
//   groups: a block owns (sequence, head, 16 value columns), sixteen lanes share two columns with their rows in
//   registers for the whole portion (8 columns and 32 lanes where blocks are few), so that a group costs one round of
//   reductions (sixteen sums over sixteen lanes share their shuffles). Operands arrive in rounds by cp.async, two rounds ahead; products and sums are packed pairs of
//   floats.
// mx_delta_step: steps in which no sequence brings more than one token. A block owns (sequence, head): the state passes
//   through registers once (a warp per group of value columns, a lane per four rows), reductions of sixteen columns
//   share their shuffles, and the norm over the head's values, its weight and the gate follow in the same kernel.
#include <math.h>

#include "conv_state.cuh"

namespace {

constexpr int DR_THREADS = 128;              // of a block of the scan
constexpr int DR_GROUP = 8;                  // tokens of a group
constexpr int DR_STAGES = 3;                 // rounds of the scan in shared memory: one computed, two on their way
// a group's numbers: T and P (a row per token), the fades from its start to each token and from each token to its end
constexpr int DR_P = DR_GROUP * DR_GROUP, DR_FADE = 2 * DR_P, DR_END = DR_FADE + DR_GROUP, DR_COEF = DR_END + DR_GROUP;

// ln(1 + e^x) without overflow on either side
__device__ __forceinline__ float softplus_exact(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

struct PrepareParams {
    const float* proj;          // rows [q | k | v | ...], `ld` floats apart
    const float* conv;          // [taps][C]
    const float* rate;          // [heads]: -exp(A_log); null: no decay per head
    const float* dt_bias;       // [heads]
    float* state;
    const int* tok_seq;
    const int* cu_q;
    const int* state_slots;
    float* qkv;                 // [tokens][C]
    float* beta;                // [tokens][heads]
    float* decay;               // [tokens][heads]
    long long state_stride;
    int ld, b_col, a_col, n_tokens, qk_heads, heads, dim, vdim, pieces;
    float q_scale, unit_eps;
};

template <int TAPS, int TOK, int NV>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const PrepareParams p) {
    pdl_trigger();
    const int lane = threadIdx.x & 31, item = blockIdx.y * 4 + (threadIdx.x >> 5), t0 = blockIdx.x * TOK;
    const int channels = 2 * p.qk_heads * p.dim + p.heads * p.vdim;
    if (item >= 2 * p.qk_heads + p.pieces) {
        if (item > 2 * p.qk_heads + p.pieces) return;
        // steps and decays of the block's tokens
        pdl_wait();
        const float* proj = after_wait(p.proj);
        for (int i = lane; i < TOK * p.heads; i += 32) {
            const int t = t0 + i / p.heads, h = i % p.heads;
            if (t >= p.n_tokens) break;
            const float* row = proj + (size_t)t * p.ld;
            p.beta[(size_t)t * p.heads + h] = 1.0f / (1.0f + expf(-row[p.b_col + h]));
            if (p.rate) p.decay[(size_t)t * p.heads + h] = expf(p.rate[h] * softplus_exact(row[p.a_col + h] + p.dt_bias[h]));
        }
        return;
    }
    const bool unit = item < 2 * p.qk_heads;
    const int col0 = unit ? item * p.dim : 2 * p.qk_heads * p.dim + (item - 2 * p.qk_heads) * 128;
    const int width = unit ? p.dim : min(128, channels - col0);
    const float scale = unit && item < p.qk_heads ? p.q_scale : 1.f;
    ConvWindow<TAPS, 4> window[NV];
    ConvVec<4> none;
#pragma unroll
    for (int e = 0; e < 4; ++e) none.v[e] = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = 4 * lane + 128 * n;
        if (c < width) window[n].weights(p.conv, channels, col0 + c);
    }
    pdl_wait();
    const float* x = after_wait(p.proj);
    int seq_before = -1;
    for (int i = 0; i < TOK; ++i) {
        const int t = t0 + i;
        if (t >= p.n_tokens) break;
        const int seq = p.tok_seq[t];
        if (seq < 0) { seq_before = -1; continue; }          // a padding row of a fixed-size batch: nobody reads it
        const int first = p.cu_q[seq];
        float* memory = p.state + (size_t)p.state_slots[seq] * p.state_stride;
        const bool alone = p.cu_q[seq + 1] - first == 1;
        ConvVec<4> y[NV];
        float squares = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = 4 * lane + 128 * n;
            if (c >= width) continue;
            if (seq != seq_before) window[n].enter(x + (size_t)first * p.ld, p.ld, memory, channels, t - first, col0 + c, none);
            y[n] = window[n].step(conv_load<4>(x + (size_t)t * p.ld + col0 + c));
            if (alone) window[n].keep(memory, channels, col0 + c);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                y[n].v[e] = silu_of<float>(y[n].v[e]);
                squares = fmaf(y[n].v[e], y[n].v[e], squares);
            }
        }
        seq_before = seq;
        float inv = 1.f;
        if (unit) inv = scale / sqrtf(warp_sum(squares) + p.unit_eps);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = 4 * lane + 128 * n;
            if (c >= width) continue;
#pragma unroll
            for (int e = 0; e < 4; ++e) y[n].v[e] *= inv;
            conv_store<4>(p.qkv + (size_t)t * channels + col0 + c, y[n]);
        }
    }
}

constexpr int DD_TOKENS = 16;      // tokens a block of the decay kernel walks with its rows of A2 in registers
constexpr int DD_CHUNK = 32;       // entries of a row of A2 a thread holds at a time

__global__ void __launch_bounds__(256)
delta_decay_kernel(const float* low, int low_ld, const float* __restrict__ a2, const float* __restrict__ dt_bias,
                   const float* __restrict__ rate, float* __restrict__ decay, int n_tokens, int channels, int dim, int rank) {
    extern __shared__ __align__(16) float low_s[];           // [DD_TOKENS][rank], rank a multiple of four
    pdl_trigger();
    const int t0 = blockIdx.x * DD_TOKENS, n_here = min(DD_TOKENS, n_tokens - t0);
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    const float* w = a2 + (size_t)min(c, channels - 1) * rank;
    float4 w4[DD_CHUNK / 4];
#pragma unroll
    for (int u = 0; u < DD_CHUNK / 4; ++u)
        w4[u] = 4 * u < rank ? *reinterpret_cast<const float4*>(w + 4 * u) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float b = c < channels ? dt_bias[c] : 0.f, r_h = c < channels ? rate[c / dim] : 0.f;
    pdl_wait();
    low = after_wait(low);
    for (int item = threadIdx.x; item < DD_TOKENS * rank; item += blockDim.x) {
        const int j = item / rank, r = item - j * rank;
        low_s[item] = j < n_here ? low[(size_t)(t0 + j) * low_ld + r] : 0.f;
    }
    __syncthreads();
    if (c >= channels) return;
    float z[DD_TOKENS];
#pragma unroll
    for (int j = 0; j < DD_TOKENS; ++j) z[j] = b;
    for (int r0 = 0; r0 < rank; r0 += DD_CHUNK) {
        if (r0 > 0) {
#pragma unroll
            for (int u = 0; u < DD_CHUNK / 4; ++u)
                w4[u] = r0 + 4 * u < rank ? *reinterpret_cast<const float4*>(w + r0 + 4 * u) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < DD_CHUNK / 4; ++u) {
            if (r0 + 4 * u < rank) {
#pragma unroll
                for (int j = 0; j < DD_TOKENS; ++j) {
                    const float4 l4 = *reinterpret_cast<const float4*>(&low_s[j * rank + r0 + 4 * u]);
                    z[j] = fmaf(w4[u].x, l4.x, z[j]); z[j] = fmaf(w4[u].y, l4.y, z[j]);
                    z[j] = fmaf(w4[u].z, l4.z, z[j]); z[j] = fmaf(w4[u].w, l4.w, z[j]);
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < DD_TOKENS; ++j)
        if (j < n_here) decay[(size_t)(t0 + j) * channels + c] = expf(r_h * softplus_exact(z[j]));
}

__device__ __forceinline__ void copy16(float* smem, const float* global, bool live) {
    const unsigned at = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = live ? 16 : 0;                         // nothing read: sixteen zero bytes
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(at), "l"(global), "r"(bytes));
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(LEFT) : "memory"); }

struct DeltaParams {
    const float* qkv;           // [tokens][C]: unit q heads | unit k heads | v heads
    const float* beta;          // [tokens][heads]
    const float* decay;         // [tokens][heads], or [tokens][heads][dim]
    float* state;               // [slots][state_stride], S at state_offset as [heads][vdim][dim]
    const int* tok_seq;
    const int* cu_q;
    const int* state_slots;
    float* out;                 // scan: [tokens][heads * vdim]
    float* coef;                // scan: [groups][heads][DR_COEF]
    float* decayed;             // scan, decays per channel: [3][tokens][heads][dim]: k, q decayed from the group's start, k to its end
    float* group_decay;         // scan, decays per channel: [groups][heads][dim]
    long long state_stride, state_offset;
    int channels, k_col, v_col, qk_heads, heads, dim, vdim, n_tokens;
};

// The group that the token `local` tokens into a sequence's portion opens or belongs to: portions start groups of their own.
__device__ __forceinline__ int group_of(int first, int seq, int local) { return (first + (DR_GROUP - 1) * seq) / DR_GROUP + local / DR_GROUP; }

// N sums over groups of LANES neighbouring lanes that share their shuffles: on return lane l of a group holds the sum number
// l / (LANES / N)
template <int N, int LANES>
__device__ __forceinline__ float shared_sums(float (&v)[N]) {
    const int lane = threadIdx.x & (LANES - 1);
    int w = LANES / 2;
#pragma unroll
    for (int n = N; n > 1; n >>= 1, w >>= 1) {
        const bool upper = lane & w;
#pragma unroll
        for (int i = 0; i < n / 2; ++i) {
            const float sent = upper ? v[i] : v[i + n / 2], kept = upper ? v[i + n / 2] : v[i];
            v[i] = kept + __shfl_xor_sync(0xffffffffu, sent, w);
        }
    }
    float sum = v[0];
#pragma unroll
    for (; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
    return sum;
}

__device__ __forceinline__ float4 times(const float4& a, const float4& b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float sum) {
    return fmaf(a.w, b.w, fmaf(a.z, b.z, fmaf(a.y, b.y, fmaf(a.x, b.x, sum))));
}

// A warp per (group of tokens, head): what the tokens of a group do to one another, whatever the state.
template <int NV, bool CHANNEL>
__global__ void __launch_bounds__(128)
delta_groups_kernel(const DeltaParams p) {
    constexpr int N = DR_GROUP, PAIRS = N * (N - 1) / 2;     // k_i k_j for i > j, then q_i k_j for i >= j: N * N sums
    static_assert(N * N == 64, "the sums of a group are two to a lane");
    __shared__ float sums_s[4][N * N];
    pdl_trigger();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, head = blockIdx.y * 4 + warp, lane = threadIdx.x & 31;
    const int seq = p.tok_seq[t];
    if (seq < 0 || head >= p.heads) return;
    const int first = p.cu_q[seq], local = t - first;
    if (local % N) return;                                   // one warp per group: the one of its first token
    const int n_here = min(N, p.cu_q[seq + 1] - t), group = group_of(first, seq, local);
    pdl_wait();
    const float* qkv = after_wait(p.qkv) + (head / (p.heads / p.qk_heads)) * p.dim;
    const float* beta_in = after_wait(p.beta);
    const float* decay = after_wait(p.decay);
    // a token that is not there: nothing fades, nothing is written
    const float my_beta = lane < n_here ? beta_in[(size_t)(t + lane) * p.heads + head] : 0.f;
    const float my_decay = !CHANNEL && lane < n_here ? decay[(size_t)(t + lane) * p.heads + head] : 1.f;
    float low[32] = {}, high[32] = {};                       // sums 0 .. 31 and 32 .. 63
    auto add = [&](int index, float v) {
        if (index < 32) low[index] += v; else high[index - 32] += v;
    };
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int r = 4 * lane + 128 * n;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), one = make_float4(1.f, 1.f, 1.f, 1.f);
        float4 k[N], q[N], g[CHANNEL ? N : 1];
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const bool live = i < n_here && r < p.dim;
            const float* row = qkv + (size_t)(t + i) * p.channels + r;
            q[i] = live ? *reinterpret_cast<const float4*>(row) : zero;
            k[i] = live ? *reinterpret_cast<const float4*>(row + p.k_col) : zero;
            if (CHANNEL)
                g[CHANNEL ? i : 0] = live ? *reinterpret_cast<const float4*>(decay + ((size_t)(t + i) * p.heads + head) * p.dim + r) : one;
        }
        const size_t plane = (size_t)p.n_tokens * p.heads * p.dim;
        float* dst = p.decayed + ((size_t)t * p.heads + head) * p.dim + r;
#pragma unroll
        for (int j = 0; j < N; ++j) {
            float4 w = k[j];                                 // the key of j as it has faded by token i
            add(PAIRS + j * (j + 1) / 2 + j, dot4(q[j], w, 0.f));
#pragma unroll
            for (int i = j + 1; i < N; ++i) {
                if (CHANNEL) w = times(w, g[CHANNEL ? i : 0]);
                add(i * (i - 1) / 2 + j, dot4(k[i], w, 0.f));
                add(PAIRS + i * (i + 1) / 2 + j, dot4(q[i], w, 0.f));
            }
            if (CHANNEL && j < n_here && r < p.dim)
                *reinterpret_cast<float4*>(dst + 2 * plane + (size_t)j * p.heads * p.dim) = w;
        }
        if (CHANNEL && r < p.dim) {
            float4 fade = one;
#pragma unroll
            for (int i = 0; i < N; ++i) {
                fade = times(fade, g[CHANNEL ? i : 0]);
                if (i >= n_here) continue;
                *reinterpret_cast<float4*>(dst + (size_t)i * p.heads * p.dim) = times(k[i], fade);
                *reinterpret_cast<float4*>(dst + plane + (size_t)i * p.heads * p.dim) = times(q[i], fade);
            }
            *reinterpret_cast<float4*>(p.group_decay + ((size_t)group * p.heads + head) * p.dim + r) = fade;
        }
    }
    float* sums = sums_s[warp];
    sums[lane] = shared_sums<32, 32>(low);
    sums[32 + lane] = shared_sums<32, 32>(high);
    __syncwarp();
    float decays[N], betas[N];                               // decays: ones where each channel has its own
#pragma unroll
    for (int i = 0; i < N; ++i) {
        decays[i] = __shfl_sync(0xffffffffu, my_decay, i);
        betas[i] = __shfl_sync(0xffffffffu, my_beta, i);
    }
    if (lane >= N) return;
    // lane j: column j of T and of P. u = T (v - S^T k, decayed) solves u_i = beta_i (v_i - .. - sum_(j<i) (k_i k_j) u_j)
    float* coef = p.coef + ((size_t)group * p.heads + head) * DR_COEF;
    float T[N];                                              // of rows lane .. N - 1
#pragma unroll
    for (int i = 0; i < N; ++i) {
        float sum = 0.f, left = 1.f;
#pragma unroll
        for (int m = i - 1; m >= 0; --m) {
            left *= decays[m + 1];                           // what is left of token m's key at token i
            if (m >= lane) sum = fmaf(sums[i * (i - 1) / 2 + m] * left, T[m], sum);
        }
        T[i] = i < lane ? 0.f : (i == lane ? betas[i] : -betas[i] * sum);
        coef[i * N + lane] = T[i];
    }
    float left = 1.f, fade = 1.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        if (i > lane) left *= decays[i];
        coef[DR_P + i * N + lane] = i >= lane ? sums[PAIRS + i * (i + 1) / 2 + min(lane, i)] * left : 0.f;
        fade *= decays[i];
        if (i == lane) coef[DR_FADE + i] = fade;
    }
    coef[DR_END + lane] = left;
}

// A round's operands. LANES lanes share two value columns, R4 groups of four rows a lane (dim <= 4 * LANES * R4): the rows
// 4 (lane + LANES u), so that their 16-byte loads are one contiguous row.
template <int LANES, int R4, int TOKENS, bool CHANNEL>
struct ScanStage {
    static constexpr int CH = 4 * LANES * R4, GROUPS = TOKENS / DR_GROUP, COLS = 2 * DR_THREADS / LANES;
    float k[TOKENS][CH], q[TOKENS][CH], k_end[CHANNEL ? TOKENS : 1][CHANNEL ? CH : 4], fade[CHANNEL ? GROUPS : 1][CHANNEL ? CH : 4];
    float v[TOKENS][COLS], coef[GROUPS][DR_COEF];
};

// Pairs of floats as the packed operations take them.
using Pair = unsigned long long;
__device__ __forceinline__ Pair fma2(Pair a, Pair b, Pair c) {
    Pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ Pair mul2(Pair a, Pair b) {
    Pair d;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ Pair both(float v) {
    Pair d;
    asm("mov.b64 %0, {%1, %1};\n" : "=l"(d) : "f"(v));
    return d;
}
__device__ __forceinline__ float sum2(Pair a) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;\n" : "=f"(x), "=f"(y) : "l"(a));
    return x + y;
}
struct Quad { Pair a, b; };                                  // four neighbouring rows
__device__ __forceinline__ Quad load_quad(const float* p) {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
    return {v.x, v.y};
}
// The same from shared memory, set out where it stands: the compiler moves no such load towards its use (with decays per
// channel it otherwise loads quad by quad and waits for each; with one per head it does better by itself).
__device__ __forceinline__ Quad ask_quad(const float* p) {
    Quad v;
    asm volatile("ld.shared.v2.b64 {%0, %1}, [%2];\n" : "=l"(v.a), "=l"(v.b) : "r"((unsigned)__cvta_generic_to_shared(p)) : "memory");
    return v;
}

template <int LANES, int R4, int TOKENS, bool CHANNEL>
__global__ void __launch_bounds__(DR_THREADS)
delta_scan_kernel(const DeltaParams p) {
    using Stage = ScanStage<LANES, R4, TOKENS, CHANNEL>;
    constexpr int COLS = Stage::COLS, PER = LANES / (2 * DR_GROUP);          // PER lanes hold the same sum of a group
    constexpr int CH = Stage::CH, ROW_THREADS = CH / 4, ROWS = DR_THREADS / ROW_THREADS;
    static_assert(DR_THREADS % ROW_THREADS == 0 && TOKENS % ROWS == 0, "a round's rows fill whole passes");
    extern __shared__ __align__(16) unsigned char scan_smem[];
    Stage* stages = reinterpret_cast<Stage*>(scan_smem);     // DR_STAGES rounds
    pdl_trigger();
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS, tid = threadIdx.x;
    const int t0 = p.cu_q[seq], t1 = p.cu_q[seq + 1];
    if (t1 <= t0) {
        // a padding sequence of a fixed-size batch, whose row bears its own number: defined output, no state
        pdl_wait();
        if (seq >= t0 && tid < COLS && col0 + tid < p.vdim)
            p.out[((size_t)seq * p.heads + head) * p.vdim + col0 + tid] = 0.f;
        return;
    }
    const int lane = tid & (LANES - 1), c = 2 * (tid / LANES), col = col0 + c;
    const int group0 = group_of(t0, seq, 0);
    float* s_base = p.state + (size_t)p.state_slots[seq] * p.state_stride + p.state_offset + ((size_t)head * p.vdim + col) * p.dim;
    Quad S[2][R4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int u = 0; u < R4; ++u) {
            const int r = 4 * (lane + LANES * u);
            S[x][u] = col + x < p.vdim && r < p.dim ? load_quad(s_base + (size_t)x * p.dim + r) : Quad{0, 0};
        }
    if (p.dim < CH) {
        // the rows that no head has stay zero in every round
        for (int i = tid; i < (int)(DR_STAGES * sizeof(Stage) / 16); i += DR_THREADS)
            reinterpret_cast<float4*>(scan_smem)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        __syncthreads();
    }
    pdl_wait();
    // a thread copies the same four rows of every ROWS-th token
    const int row_j = tid / ROW_THREADS, r0 = (tid % ROW_THREADS) * 4;
    const bool copies = r0 < p.dim;
    const size_t plane = (size_t)p.n_tokens * p.heads * p.dim, row_stride = CHANNEL ? (size_t)p.heads * p.dim : (size_t)p.channels;
    const float* k_from = CHANNEL ? after_wait(p.decayed) + ((size_t)t0 * p.heads + head) * p.dim + r0
                                  : after_wait(p.qkv) + (size_t)t0 * p.channels + p.k_col + (head / (p.heads / p.qk_heads)) * p.dim + r0;
    const float* q_from = CHANNEL ? k_from + plane : k_from - p.k_col;
    const float* v_from = after_wait(p.qkv) + (size_t)t0 * p.channels + p.v_col + head * p.vdim + col0;
    const float* coef = after_wait(p.coef) + ((size_t)group0 * p.heads + head) * DR_COEF;
    const float* group_decay = after_wait(p.group_decay) + ((size_t)group0 * p.heads + head) * p.dim;
    const int n = t1 - t0;
    auto fetch = [&](Stage& s, int base) {                   // tokens base .. of the portion; an empty group when there are none
        if (base < n) {
            const bool whole = base + TOKENS <= n;
            if (copies) {
                const size_t at = (size_t)(base + row_j) * row_stride;
                const float *k_at = k_from + at, *q_at = q_from + at;
#pragma unroll
                for (int j = 0; j < TOKENS; j += ROWS) {
                    const bool live = whole || base + row_j + j < n;
                    const float *k = live ? k_at : k_from, *q = live ? q_at : q_from;
                    copy16(&s.k[row_j + j][r0], k, live);
                    copy16(&s.q[row_j + j][r0], q, live);
                    if (CHANNEL) copy16(&s.k_end[CHANNEL ? row_j + j : 0][CHANNEL ? r0 : 0], k + 2 * plane, live);
                    k_at += ROWS * row_stride;
                    q_at += ROWS * row_stride;
                }
            }
            if (tid < TOKENS * (COLS / 4)) {
                const int j = tid / (COLS / 4), e = (tid % (COLS / 4)) * 4;
                const bool live = base + j < n && col0 + e < p.vdim;
                copy16(&s.v[j][e], live ? v_from + (size_t)(base + j) * p.channels + e : v_from, live);
            }
            const int group = base / DR_GROUP, groups = (n - base + DR_GROUP - 1) / DR_GROUP;
#pragma unroll
            for (int g = 0; g < Stage::GROUPS; ++g) {
                if (tid < DR_COEF / 4)
                    copy16(&s.coef[g][4 * tid], coef + (size_t)(group + (g < groups ? g : 0)) * p.heads * DR_COEF + 4 * tid, g < groups);
                if (CHANNEL && row_j == (g + 1) % ROWS && copies)
                    copy16(&s.fade[CHANNEL ? g : 0][CHANNEL ? r0 : 0],
                           group_decay + (size_t)(group + (g < groups ? g : 0)) * p.heads * p.dim + r0, g < groups);
            }
        }
        copies_commit();
    };
    // the one of the group's sums that a lane ends up with: token own_i, column own_x
    const int own_i = lane / (2 * PER), own_x = lane / PER & 1;
    const bool writes = lane % PER == 0 && col + own_x < p.vdim;
    const size_t out_stride = (size_t)p.heads * p.vdim;
    float* out = p.out + ((size_t)(t0 + own_i) * p.heads + head) * p.vdim + col + own_x;
    auto advance = [&](const Stage& s, int g, int t) {
        const int j0 = g * DR_GROUP;
        const float* numbers = s.coef[g];
        Pair pairs[2 * DR_GROUP];
        float sums[2 * DR_GROUP];
        Quad k[DR_GROUP][R4];
        auto ask = [&](Quad (&into)[DR_GROUP][R4], const float (*rows)[CH]) {
#pragma unroll
            for (int i = 0; i < DR_GROUP; ++i)
#pragma unroll
                for (int u = 0; u < R4; ++u) into[i][u] = ask_quad(&rows[j0 + i][4 * (lane + LANES * u)]);
        };
        // both columns' sums over the lane's rows for the rows of `rows` (with one decay per head: kept in `kept`)
        auto contract = [&](const float (*rows)[CH], const Quad (&asked)[DR_GROUP][R4], Quad (*kept)[R4]) {
#pragma unroll
            for (int i = 0; i < 2 * DR_GROUP; ++i) pairs[i] = 0;
            if constexpr (CHANNEL) {
#pragma unroll
                for (int u = 0; u < R4; ++u) {
#pragma unroll
                    for (int i = 0; i < DR_GROUP; ++i) {
                        pairs[2 * i] = fma2(S[0][u].a, asked[i][u].a, pairs[2 * i]);
                        pairs[2 * i + 1] = fma2(S[1][u].a, asked[i][u].a, pairs[2 * i + 1]);
                    }
#pragma unroll
                    for (int i = 0; i < DR_GROUP; ++i) {
                        pairs[2 * i] = fma2(S[0][u].b, asked[i][u].b, pairs[2 * i]);
                        pairs[2 * i + 1] = fma2(S[1][u].b, asked[i][u].b, pairs[2 * i + 1]);
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < DR_GROUP; ++i)
#pragma unroll
                    for (int u = 0; u < R4; ++u) {
                        const Quad m = load_quad(&rows[j0 + i][4 * (lane + LANES * u)]);
                        pairs[2 * i] = fma2(S[0][u].b, m.b, fma2(S[0][u].a, m.a, pairs[2 * i]));
                        pairs[2 * i + 1] = fma2(S[1][u].b, m.b, fma2(S[1][u].a, m.a, pairs[2 * i + 1]));
                        if (kept) kept[i][u] = m;
                    }
            }
#pragma unroll
            for (int i = 0; i < 2 * DR_GROUP; ++i) sums[i] = sum2(pairs[i]);
        };
        Quad q[DR_GROUP][R4];
        if constexpr (CHANNEL) ask(k, s.k);
        const float my_fade = CHANNEL ? 1.f : numbers[DR_FADE + own_i];
        const float my_v = s.v[j0 + own_i][c + own_x];
        if constexpr (CHANNEL) ask(q, s.q);
        contract(s.k, k, CHANNEL ? nullptr : k);
        // v - S^T k of the lane's own token and column, then its row of T times those of the group
        const float mine = fmaf(-my_fade, shared_sums<2 * DR_GROUP, LANES>(sums), my_v);
        contract(s.q, q, nullptr);
        if constexpr (CHANNEL) ask(k, s.k_end);
        float write[2] = {0.f, 0.f};
#pragma unroll
        for (int j = 0; j < DR_GROUP; j += 4) {
            const float4 row = *reinterpret_cast<const float4*>(&numbers[own_i * DR_GROUP + j]);
            write[0] = fmaf(row.x, __shfl_sync(0xffffffffu, mine, PER * (2 * j + own_x), LANES), write[0]);
            write[1] = fmaf(row.y, __shfl_sync(0xffffffffu, mine, PER * (2 * j + 2 + own_x), LANES), write[1]);
            write[0] = fmaf(row.z, __shfl_sync(0xffffffffu, mine, PER * (2 * j + 4 + own_x), LANES), write[0]);
            write[1] = fmaf(row.w, __shfl_sync(0xffffffffu, mine, PER * (2 * j + 6 + own_x), LANES), write[1]);
        }
        const float my_write = write[0] + write[1];
        float w[DR_GROUP][2];
#pragma unroll
        for (int i = 0; i < DR_GROUP; ++i) {
            w[i][0] = __shfl_sync(0xffffffffu, my_write, PER * 2 * i, LANES);
            w[i][1] = __shfl_sync(0xffffffffu, my_write, PER * (2 * i + 1), LANES);
        }
        const float my_seen = shared_sums<2 * DR_GROUP, LANES>(sums);
        // o = S^T q + P u
        float o[2] = {my_fade * my_seen, 0.f};
#pragma unroll
        for (int j = 0; j < DR_GROUP; j += 4) {
            const float4 row = *reinterpret_cast<const float4*>(&numbers[DR_P + own_i * DR_GROUP + j]);
            o[0] = fmaf(row.x, own_x ? w[j][1] : w[j][0], o[0]);
            o[1] = fmaf(row.y, own_x ? w[j + 1][1] : w[j + 1][0], o[1]);
            o[0] = fmaf(row.z, own_x ? w[j + 2][1] : w[j + 2][0], o[0]);
            o[1] = fmaf(row.w, own_x ? w[j + 3][1] : w[j + 3][0], o[1]);
        }
        if (writes && t + own_i < n) out[(size_t)t * out_stride] = o[0] + o[1];
        // the state at the group's end
        if (!CHANNEL) {
            const Pair fade = both(numbers[DR_FADE + DR_GROUP - 1]);
#pragma unroll
            for (int i = 0; i < DR_GROUP; i += 4) {
                const float4 end = *reinterpret_cast<const float4*>(&numbers[DR_END + i]);
                w[i][0] *= end.x; w[i][1] *= end.x; w[i + 1][0] *= end.y; w[i + 1][1] *= end.y;
                w[i + 2][0] *= end.z; w[i + 2][1] *= end.z; w[i + 3][0] *= end.w; w[i + 3][1] *= end.w;
            }
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int u = 0; u < R4; ++u) S[x][u] = {mul2(S[x][u].a, fade), mul2(S[x][u].b, fade)};
        } else {
#pragma unroll
            for (int u = 0; u < R4; ++u) {
                const Quad f = load_quad(&s.fade[CHANNEL ? g : 0][CHANNEL ? 4 * (lane + LANES * u) : 0]);
#pragma unroll
                for (int x = 0; x < 2; ++x) S[x][u] = {mul2(S[x][u].a, f.a), mul2(S[x][u].b, f.b)};
            }
        }
#pragma unroll
        for (int i = 0; i < DR_GROUP; ++i) {
            const Pair w0 = both(w[i][0]), w1 = both(w[i][1]);
#pragma unroll
            for (int u = 0; u < R4; ++u) {
                const Quad e = k[i][u];
                S[0][u] = {fma2(e.a, w0, S[0][u].a), fma2(e.b, w0, S[0][u].b)};
                S[1][u] = {fma2(e.a, w1, S[1][u].a), fma2(e.b, w1, S[1][u].b)};
            }
        }
    };
    fetch(stages[0], 0);
    fetch(stages[1], TOKENS);
    int at = 0;
    for (int base = 0; base < n; base += TOKENS) {
        copies_wait<1>();
        __syncthreads();                                     // the round is there, the one before it is done with
        fetch(stages[at == 0 ? DR_STAGES - 1 : at - 1], base + 2 * TOKENS);
        const int groups = min(Stage::GROUPS, (n - base + DR_GROUP - 1) / DR_GROUP);
        for (int g = 0; g < groups; ++g) advance(stages[at], g, base + g * DR_GROUP);
        at = at == DR_STAGES - 1 ? 0 : at + 1;
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int u = 0; u < R4; ++u) {
            const int r = 4 * (lane + LANES * u);
            if (col + x < p.vdim && r < p.dim)
                *reinterpret_cast<ulonglong2*>(s_base + (size_t)x * p.dim + r) = make_ulonglong2(S[x][u].a, S[x][u].b);
        }
}

struct StepParams {
    DeltaParams d;
    const float* gate;          // rows gate_ld floats apart: [heads * vdim] logits
    const float* weight;        // [vdim]
    int gate_ld, out_ld, sigmoid_gate, true_vdim;
    float eps, out_scale;
};

template <typename T, int NV, bool CHANNEL>
__global__ void __launch_bounds__(256)
delta_step_kernel(const StepParams sp, T* __restrict__ out) {
    constexpr int COLS = NV == 1 ? 16 : 8, PER = 32 / COLS;  // value columns of a warp's group, lanes that hold one's sum
    extern __shared__ float o_s[];                           // [vdim]
    __shared__ float scratch[32];
    pdl_trigger();
    const DeltaParams& p = sp.d;
    const int seq = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = p.cu_q[seq];
    if (p.cu_q[seq + 1] <= t) {
        pdl_wait();
        if (seq >= t)
            for (int e = threadIdx.x; e < p.vdim; e += 256)
                out[(size_t)seq * sp.out_ld + (size_t)head * p.vdim + e] = from_float<T>(0.f);
        return;
    }
    float* s_head = p.state + (size_t)p.state_slots[seq] * p.state_stride + p.state_offset + (size_t)head * p.vdim * p.dim;
    float4 S[COLS][NV];
    auto load = [&](int e0) {
#pragma unroll
        for (int x = 0; x < COLS; ++x)
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int r = 4 * lane + 128 * n;
                S[x][n] = e0 + x < p.vdim && r < p.dim ? *reinterpret_cast<const float4*>(s_head + (size_t)(e0 + x) * p.dim + r)
                                                       : make_float4(0.f, 0.f, 0.f, 0.f);
            }
    };
    load(warp * COLS);                                       // the state is what earlier steps left
    pdl_wait();
    const float* row = after_wait(p.qkv) + (size_t)t * p.channels + (head / (p.heads / p.qk_heads)) * p.dim;
    const float* v_row = after_wait(p.qkv) + (size_t)t * p.channels + p.v_col + (size_t)head * p.vdim;
    const float* decay = after_wait(p.decay);
    const float beta = after_wait(p.beta)[(size_t)t * p.heads + head];
    float4 q[NV], k[NV], g[NV];
    float kq = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int r = 4 * lane + 128 * n;
        const bool live = r < p.dim;
        q[n] = live ? *reinterpret_cast<const float4*>(row + r) : make_float4(0.f, 0.f, 0.f, 0.f);
        k[n] = live ? *reinterpret_cast<const float4*>(row + p.k_col + r) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (CHANNEL) {
            g[n] = live ? *reinterpret_cast<const float4*>(decay + ((size_t)t * p.heads + head) * p.dim + r)
                        : make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
            const float g1 = decay[(size_t)t * p.heads + head];
            g[n] = make_float4(g1, g1, g1, g1);
        }
        kq += (k[n].x * q[n].x + k[n].y * q[n].y) + (k[n].z * q[n].z + k[n].w * q[n].w);
    }
    kq = warp_sum(kq);
    for (int e0 = warp * COLS; e0 < p.vdim; e0 += 8 * COLS) {
        if (e0 != warp * COLS) load(e0);
        float held[COLS], seen[COLS];
#pragma unroll
        for (int x = 0; x < COLS; ++x) {
            held[x] = seen[x] = 0.f;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                float4& s = S[x][n];
                s.x *= g[n].x; s.y *= g[n].y; s.z *= g[n].z; s.w *= g[n].w;
                held[x] += fmaf(s.x, k[n].x, s.y * k[n].y) + fmaf(s.z, k[n].z, s.w * k[n].w);
                seen[x] += fmaf(s.x, q[n].x, s.y * q[n].y) + fmaf(s.z, q[n].z, s.w * q[n].w);
            }
        }
        const float sum_k = shared_sums<COLS, 32>(held), sum_q = shared_sums<COLS, 32>(seen);
        const int mine = e0 + lane / PER;
        const float write = mine < p.vdim ? beta * (v_row[mine] - sum_k) : 0.f;
        // S^T q after the write: what the forgetting state gives plus the write times k . q
        if (lane % PER == 0 && mine < p.vdim) o_s[mine] = fmaf(write, kq, sum_q);
#pragma unroll
        for (int x = 0; x < COLS; ++x) {
            const float u = __shfl_sync(0xffffffffu, write, x * PER);
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int r = 4 * lane + 128 * n;
                float4& s = S[x][n];
                s.x = fmaf(k[n].x, u, s.x); s.y = fmaf(k[n].y, u, s.y); s.z = fmaf(k[n].z, u, s.z); s.w = fmaf(k[n].w, u, s.w);
                if (e0 + x < p.vdim && r < p.dim) *reinterpret_cast<float4*>(s_head + (size_t)(e0 + x) * p.dim + r) = s;
            }
        }
    }
    __syncthreads();
    float squares = 0.f;
    for (int e = threadIdx.x; e < p.vdim; e += 256) squares = fmaf(o_s[e], o_s[e], squares);
    const float inv = sp.out_scale / sqrtf(block_sum(squares, scratch) / (float)sp.true_vdim + sp.eps);
    const float* gate = after_wait(sp.gate) + (size_t)t * sp.gate_ld + (size_t)head * p.vdim;
    for (int e = threadIdx.x; e < p.vdim; e += 256) {
        const float z = gate[e], s = 1.f / (1.f + expf(-z));
        out[(size_t)t * sp.out_ld + (size_t)head * p.vdim + e] =
            from_float<T>(o_s[e] * inv * sp.weight[e] * (sp.sigmoid_gate ? s : z * s));
    }
}

template <int TAPS, int NV>
void launch_prepare(const PrepareParams& p, cudaStream_t stream) {
    const int items = 2 * p.qk_heads + p.pieces + 1;
    // few tokens: a warp's walk would be the whole latency; many: neighbouring tokens share their inputs
    if (p.n_tokens <= 256)
        mx_launch_chained(delta_prepare_kernel<TAPS, 1, NV>, dim3(p.n_tokens, (items + 3) / 4), dim3(128), 0, stream, p);
    else
        mx_launch_chained(delta_prepare_kernel<TAPS, 8, NV>, dim3((p.n_tokens + 7) / 8, (items + 3) / 4), dim3(128), 0, stream, p);
}

template <int LANES, int R4, int TOKENS, bool CHANNEL>
int launch_walk(const DeltaParams& p, int n_seqs, cudaStream_t stream) {
    constexpr size_t smem = DR_STAGES * sizeof(ScanStage<LANES, R4, TOKENS, CHANNEL>);
    constexpr int COLS = ScanStage<LANES, R4, TOKENS, CHANNEL>::COLS;
    static bool ready = false;
    if (!ready) {
        if (cudaFuncSetAttribute(delta_scan_kernel<LANES, R4, TOKENS, CHANNEL>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)smem) != cudaSuccess)
            MX_REFUSE("delta rule: cannot reserve %zu bytes of shared memory", smem);
        ready = true;
    }
    mx_launch_chained(delta_scan_kernel<LANES, R4, TOKENS, CHANNEL>, dim3(n_seqs, p.heads, (p.vdim + COLS - 1) / COLS),
                      dim3(DR_THREADS), smem, stream, p);
    return mx_launch_status();
}

template <bool CHANNEL>
int launch_scan(const DeltaParams& p, int n_seqs, int sms, cudaStream_t stream) {
    const dim3 grid(p.n_tokens, (p.heads + 3) / 4);
    if (p.dim <= 128) mx_launch_chained(delta_groups_kernel<1, CHANNEL>, grid, dim3(128), 0, stream, p);
    else mx_launch_chained(delta_groups_kernel<2, CHANNEL>, grid, dim3(128), 0, stream, p);
    // few columns: twice as many lanes to a column shorten each walk, as long as no SM gets two of the then twice as many
    // blocks (2,048 tokens x 8 heads of 128 x 128: 218 -> 196 us; at 16 heads 224 -> 251)
    const long long blocks = (long long)n_seqs * p.heads * ((p.vdim + 15) / 16);
    const bool wide = p.dim > 64 && 2 * blocks <= sms;
    if (p.dim <= 64) return launch_walk<16, 1, 16, CHANNEL>(p, n_seqs, stream);
    if (p.dim <= 128)
        return wide ? launch_walk<32, 1, 16, CHANNEL>(p, n_seqs, stream) : launch_walk<16, 2, 16, CHANNEL>(p, n_seqs, stream);
    return wide ? launch_walk<32, 2, 8, CHANNEL>(p, n_seqs, stream) : launch_walk<16, 4, 8, CHANNEL>(p, n_seqs, stream);
}

const char* delta_sizes(int qk_heads, int heads, int dim, int vdim) {
    if (dim <= 0 || dim > 256 || dim % 4 || vdim <= 0 || vdim % 4) return "head sizes (multiples of four, keys of at most 256)";
    if (qk_heads <= 0 || heads <= 0 || heads % qk_heads || heads > 65535) return "head counts";
    return nullptr;
}

}  // namespace

extern "C" int mx_delta_prepare(const float* proj, int ld, int b_col, int a_col, const float* conv, int taps, const float* rate,
                                const float* dt_bias, float* state, long long state_stride, const int* tok_seq,
                                const int* cu_q, const int* state_slots, float* qkv, float* beta, float* decay, int n_tokens,
                                int qk_heads, int heads, int dim, int vdim, float q_scale, float unit_eps, cudaStream_t stream) {
    if (n_tokens <= 0) return MX_OK;
    if (const char* what = delta_sizes(qk_heads, heads, dim, vdim)) MX_REFUSE("delta rule: %s: %d of %d, %d of %d", what, qk_heads, dim, heads, vdim);
    const int channels = 2 * qk_heads * dim + heads * vdim;
    if (ld < channels || ld % 4 || state_stride % 4 || state_stride < (long long)(taps - 1) * channels)
        MX_REFUSE("delta rule: rows of %d floats or a state of %lld floats do not fit %d channels", ld, state_stride, channels);
    if (((uintptr_t)proj | (uintptr_t)conv | (uintptr_t)state | (uintptr_t)qkv) % 16) MX_REFUSE("delta rule: unaligned operands");
    PrepareParams p;
    p.proj = proj; p.conv = conv; p.rate = rate; p.dt_bias = dt_bias; p.state = state; p.tok_seq = tok_seq; p.cu_q = cu_q;
    p.state_slots = state_slots; p.qkv = qkv; p.beta = beta; p.decay = decay; p.state_stride = state_stride; p.ld = ld;
    p.b_col = b_col; p.a_col = a_col; p.n_tokens = n_tokens; p.qk_heads = qk_heads; p.heads = heads; p.dim = dim; p.vdim = vdim;
    p.pieces = (heads * vdim + 127) / 128; p.q_scale = q_scale; p.unit_eps = unit_eps;
#define MX_PREPARE(TAPS) (dim <= 128 ? launch_prepare<TAPS, 1>(p, stream) : launch_prepare<TAPS, 2>(p, stream))
    switch (taps) {
        case 2: MX_PREPARE(2); break;
        case 3: MX_PREPARE(3); break;
        case 4: MX_PREPARE(4); break;
        case 8: MX_PREPARE(8); break;
        case 16: MX_PREPARE(16); break;
        default: MX_REFUSE("delta rule: a convolution of %d taps (2, 3, 4, 8 or 16; shorter ones are filled up with zeros)", taps);
    }
#undef MX_PREPARE
    return mx_launch_status();
}

extern "C" int mx_delta_decay(const float* low, int low_ld, const float* a2, const float* dt_bias, const float* rate,
                              float* decay, int n_tokens, int channels, int dim, int rank, cudaStream_t stream) {
    if (n_tokens <= 0) return MX_OK;
    const size_t smem = (size_t)DD_TOKENS * rank * sizeof(float);
    if (rank <= 0 || rank % 4 || smem > 48 * 1024) MX_REFUSE("delta rule: a decay rank of %d (a multiple of four up to 768)", rank);
    if (channels <= 0 || dim <= 0 || (uintptr_t)a2 % 16) MX_REFUSE("delta rule: %d decays of heads of %d", channels, dim);
    mx_launch_chained(delta_decay_kernel, dim3((n_tokens + DD_TOKENS - 1) / DD_TOKENS, (channels + 255) / 256), dim3(256), smem,
                      stream, low, low_ld, a2, dt_bias, rate, decay, n_tokens, channels, dim, rank);
    return mx_launch_status();
}

static int delta_params(DeltaParams& p, const float* qkv, const float* beta, const float* decay, float* state,
                        long long state_stride, long long state_offset, const int* cu_q, const int* state_slots,
                        int qk_heads, int heads, int dim, int vdim) {
    if (const char* what = delta_sizes(qk_heads, heads, dim, vdim)) MX_REFUSE("delta rule: %s: %d of %d, %d of %d", what, qk_heads, dim, heads, vdim);
    if (state_stride % 4 || state_offset % 4 || state_stride < state_offset + (long long)heads * dim * vdim)
        MX_REFUSE("delta rule: a state of %lld floats from %lld is too short", state_stride, state_offset);
    if (((uintptr_t)qkv | (uintptr_t)decay | (uintptr_t)state) % 16) MX_REFUSE("delta rule: unaligned operands");
    p.qkv = qkv; p.beta = beta; p.decay = decay; p.state = state; p.cu_q = cu_q; p.state_slots = state_slots;
    p.tok_seq = nullptr; p.out = p.coef = p.decayed = p.group_decay = nullptr; p.n_tokens = 0; p.state_stride = state_stride; p.state_offset = state_offset; p.channels = 2 * qk_heads * dim + heads * vdim;
    p.k_col = qk_heads * dim; p.v_col = 2 * qk_heads * dim; p.qk_heads = qk_heads; p.heads = heads; p.dim = dim; p.vdim = vdim;
    return MX_OK;
}

// How many floats mx_delta_scan wants as scratch.
extern "C" long long mx_delta_scan_scratch(int per_channel, int n_tokens, int n_seqs, int heads, int dim) {
    const long long groups = (n_tokens + (long long)(DR_GROUP - 1) * n_seqs) / DR_GROUP + 1;
    return groups * heads * DR_COEF + (per_channel ? (3LL * n_tokens + groups) * heads * dim : 0);
}

// `per_channel`: decay is [tokens][heads][dim] instead of [tokens][heads]
extern "C" int mx_delta_scan(const float* qkv, const float* beta, const float* decay, int per_channel, float* state,
                             long long state_stride, long long state_offset, const int* tok_seq, const int* cu_q,
                             const int* state_slots, float* scratch, float* out, int n_tokens, int n_seqs, int qk_heads,
                             int heads, int dim, int vdim, cudaStream_t stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return MX_OK;
    DeltaParams p;
    const int rc = delta_params(p, qkv, beta, decay, state, state_stride, state_offset, cu_q, state_slots, qk_heads, heads, dim,
                                vdim);
    if (rc != MX_OK) return rc;
    if ((uintptr_t)scratch % 16) MX_REFUSE("delta rule: unaligned scratch memory");
    const long long groups = (n_tokens + (long long)(DR_GROUP - 1) * n_seqs) / DR_GROUP + 1;
    p.tok_seq = tok_seq; p.out = out; p.n_tokens = n_tokens; p.coef = scratch;
    p.group_decay = scratch + groups * heads * DR_COEF;
    p.decayed = p.group_decay + groups * heads * dim;
    static int sms = 0;
    if (sms == 0) {
        int device = 0;
        cudaGetDevice(&device);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
    }
    return per_channel ? launch_scan<true>(p, n_seqs, sms, stream) : launch_scan<false>(p, n_seqs, sms, stream);
}

// The scan of steps without a sequence of more than one token, with what follows it:
// out[t][h][e] = out_scale * o[h][e] / sqrt(mean_e(o^2) + eps) * weight[e] * act(gate[t][h][e]), act silu or sigmoid.
extern "C" int mx_delta_step(const float* qkv, const float* beta, const float* decay, int per_channel, float* state,
                             long long state_stride, long long state_offset, const int* cu_q, const int* state_slots,
                             const float* gate, int gate_ld, int sigmoid_gate, const float* weight, float eps, float out_scale,
                             void* out, int dtype, int out_ld, int n_seqs, int qk_heads, int heads, int dim, int vdim,
                             int true_vdim, cudaStream_t stream) {
    if (n_seqs <= 0) return MX_OK;
    StepParams sp;
    const int rc = delta_params(sp.d, qkv, beta, decay, state, state_stride, state_offset, cu_q, state_slots, qk_heads, heads,
                                dim, vdim);
    if (rc != MX_OK) return rc;
    if (true_vdim <= 0 || true_vdim > vdim || vdim > 12 * 1024) MX_REFUSE("delta rule: heads of %d values in %d", true_vdim, vdim);
    sp.gate = gate; sp.weight = weight; sp.gate_ld = gate_ld; sp.out_ld = out_ld; sp.sigmoid_gate = sigmoid_gate;
    sp.true_vdim = true_vdim; sp.eps = eps; sp.out_scale = out_scale;
    const dim3 grid(n_seqs, heads);
    const size_t smem = (size_t)vdim * sizeof(float);
#define MX_STEP(T, NV, CHANNEL) mx_launch_chained(delta_step_kernel<T, NV, CHANNEL>, grid, dim3(256), smem, stream, sp, (T*)out)
#define MX_STEP_DTYPE(NV, CHANNEL)                                     \
    do {                                                               \
        if (dtype == MX_DTYPE_F32) MX_STEP(float, NV, CHANNEL);        \
        else MX_STEP(__nv_bfloat16, NV, CHANNEL);                      \
    } while (0)
    if (dim <= 128) {
        if (per_channel) MX_STEP_DTYPE(1, true); else MX_STEP_DTYPE(1, false);
    } else {
        if (per_channel) MX_STEP_DTYPE(2, true); else MX_STEP_DTYPE(2, false);
    }
#undef MX_STEP_DTYPE
#undef MX_STEP
    return mx_launch_status();
}
