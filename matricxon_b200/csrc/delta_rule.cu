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
// mx_delta_scan: every sequence's tokens in order. A block owns (sequence, head, 16 value columns); eight lanes share a
//   column, each with an eighth of its rows in registers for the whole portion. Tokens arrive in rounds by cp.async, two
//   rounds in flight; S^T k is reduced by three shuffles a token, the shares of the read-outs meet in shared memory once a
//   round.
// mx_delta_step: steps in which no sequence brings more than one token. A block owns (sequence, head): the state passes
//   through registers once (a warp per group of value columns, a lane per four rows), reductions of sixteen columns
//   share their shuffles, and the norm over the head's values, its weight and the gate follow in the same kernel.
#include <math.h>

#include "conv_state.cuh"

namespace {

constexpr int DR_COLS = 16, DR_LANES = 8, DR_THREADS = DR_COLS * DR_LANES;

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
__device__ __forceinline__ void copy4(float* smem, const float* global, bool live) {
    const unsigned at = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = live ? 4 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(at), "l"(global), "r"(bytes));
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(LEFT) : "memory"); }

struct DeltaParams {
    const float* qkv;           // [tokens][C]: unit q heads | unit k heads | v heads
    const float* beta;          // [tokens][heads]
    const float* decay;         // [tokens][heads], or [tokens][heads][dim]
    float* state;               // [slots][state_stride], S at state_offset as [heads][vdim][dim]
    const int* cu_q;
    const int* state_slots;
    float* out;                 // scan: [tokens][heads * vdim]
    long long state_stride, state_offset;
    int channels, k_col, v_col, qk_heads, heads, dim, vdim;
};

// ROWS rows of a column a lane (dim <= 8 * ROWS): the groups of four rows 4 (lane + 8 u), so that eight lanes' 16-byte
// loads are one contiguous row
template <int ROWS, int TOKENS, bool CHANNEL>
struct ScanStage {
    static constexpr int CH = DR_LANES * ROWS;
    float k[TOKENS][CH], q[TOKENS][CH], g[CHANNEL ? TOKENS : 1][CHANNEL ? CH : 4], v[TOKENS][DR_COLS], beta[TOKENS], g1[TOKENS];
};

template <int ROWS, int TOKENS, bool CHANNEL>
__global__ void __launch_bounds__(DR_THREADS)
delta_scan_kernel(const DeltaParams p) {
    using Stage = ScanStage<ROWS, TOKENS, CHANNEL>;
    constexpr int CH = Stage::CH, R4 = ROWS / 4;
    extern __shared__ __align__(16) unsigned char scan_smem[];
    Stage* stages = reinterpret_cast<Stage*>(scan_smem);     // two rounds in flight
    __shared__ float o_s[TOKENS][DR_LANES][DR_COLS];
    pdl_trigger();
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * DR_COLS, tid = threadIdx.x;
    const int t0 = p.cu_q[seq], t1 = p.cu_q[seq + 1];
    if (t1 <= t0) {
        // a padding sequence of a fixed-size batch, whose row bears its own number: defined output, no state
        pdl_wait();
        if (seq >= t0 && tid < DR_COLS && col0 + tid < p.vdim)
            p.out[((size_t)seq * p.heads + head) * p.vdim + col0 + tid] = 0.f;
        return;
    }
    const int lane = tid & (DR_LANES - 1), c = tid / DR_LANES, col = col0 + c;
    const int qk_head = head / (p.heads / p.qk_heads);
    const bool live_col = col < p.vdim;
    float* s_base = p.state + (size_t)p.state_slots[seq] * p.state_stride + p.state_offset + ((size_t)head * p.vdim + col) * p.dim;
    float4 S[R4];
#pragma unroll
    for (int u = 0; u < R4; ++u) {
        const int r = 4 * (lane + DR_LANES * u);
        S[u] = live_col && r < p.dim ? *reinterpret_cast<const float4*>(s_base + r) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    const float* qkv = after_wait(p.qkv);
    const float* beta = after_wait(p.beta);
    const float* decay = after_wait(p.decay);
    auto fetch = [&](Stage& s, int base) {
        for (int item = tid; item < TOKENS * (CH / 4); item += DR_THREADS) {
            const int j = item / (CH / 4), r = (item % (CH / 4)) * 4, t = min(base + j, t1 - 1);
            const bool live = base + j < t1 && r < p.dim;
            const float* row = qkv + (size_t)t * p.channels + qk_head * p.dim + (r < p.dim ? r : 0);
            copy16(&s.q[j][r], row, live);
            copy16(&s.k[j][r], row + p.k_col, live);
            if (CHANNEL) copy16(&s.g[CHANNEL ? j : 0][CHANNEL ? r : 0],
                                decay + ((size_t)t * p.heads + head) * p.dim + (r < p.dim ? r : 0), live);
        }
        for (int item = tid; item < TOKENS * (DR_COLS / 4); item += DR_THREADS) {
            const int j = item / (DR_COLS / 4), e = (item % (DR_COLS / 4)) * 4, t = min(base + j, t1 - 1);
            const bool live = base + j < t1 && col0 + e < p.vdim;
            copy16(&s.v[j][e], qkv + (size_t)t * p.channels + p.v_col + head * p.vdim + (col0 + e < p.vdim ? col0 + e : 0), live);
        }
        if (tid < TOKENS) {
            const int t = min(base + tid, t1 - 1);
            copy4(&s.beta[tid], beta + (size_t)t * p.heads + head, base + tid < t1);
            if (!CHANNEL) copy4(&s.g1[tid], decay + (size_t)t * p.heads + head, base + tid < t1);
        }
        copies_commit();
    };
    struct Operands {
        float4 k[R4], q[R4], g[CHANNEL ? R4 : 1];
        float v, beta, g1;
    };
    auto read = [&](Operands& into, const Stage& s, int j) {
#pragma unroll
        for (int u = 0; u < R4; ++u) {
            const int r = 4 * (lane + DR_LANES * u);
            into.k[u] = *reinterpret_cast<const float4*>(&s.k[j][r]);
            into.q[u] = *reinterpret_cast<const float4*>(&s.q[j][r]);
            if (CHANNEL) into.g[CHANNEL ? u : 0] = *reinterpret_cast<const float4*>(&s.g[CHANNEL ? j : 0][CHANNEL ? r : 0]);
        }
        into.v = s.v[j][c];
        into.beta = s.beta[j];
        into.g1 = CHANNEL ? 1.f : s.g1[j];
    };
    auto advance = [&](const Operands& now, int j) {
        float4 held = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < R4; ++u) {
            const float4 g = CHANNEL ? now.g[CHANNEL ? u : 0] : make_float4(now.g1, now.g1, now.g1, now.g1);
            S[u].x *= g.x; S[u].y *= g.y; S[u].z *= g.z; S[u].w *= g.w;
            held.x = fmaf(S[u].x, now.k[u].x, held.x); held.y = fmaf(S[u].y, now.k[u].y, held.y);
            held.z = fmaf(S[u].z, now.k[u].z, held.z); held.w = fmaf(S[u].w, now.k[u].w, held.w);
        }
        float sum = (held.x + held.y) + (held.z + held.w);
#pragma unroll
        for (int o = DR_LANES / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        const float write = now.beta * (now.v - sum);
        float4 read_out = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < R4; ++u) {
            S[u].x = fmaf(now.k[u].x, write, S[u].x); S[u].y = fmaf(now.k[u].y, write, S[u].y);
            S[u].z = fmaf(now.k[u].z, write, S[u].z); S[u].w = fmaf(now.k[u].w, write, S[u].w);
            read_out.x = fmaf(S[u].x, now.q[u].x, read_out.x); read_out.y = fmaf(S[u].y, now.q[u].y, read_out.y);
            read_out.z = fmaf(S[u].z, now.q[u].z, read_out.z); read_out.w = fmaf(S[u].w, now.q[u].w, read_out.w);
        }
        o_s[j][lane][c] = (read_out.x + read_out.y) + (read_out.z + read_out.w);
    };
    fetch(stages[0], t0);
    int at = 0;
    for (int base = t0; base < t1; base += TOKENS, at ^= 1) {
        const int n_here = min(TOKENS, t1 - base);
        if (base + TOKENS < t1) {
            fetch(stages[at ^ 1], base + TOKENS);
            copies_wait<1>();
        } else {
            copies_wait<0>();
        }
        __syncthreads();
        const Stage& s = stages[at];
        Operands even, odd;
        read(even, s, 0);
        for (int j = 0; j < n_here; j += 2) {
            if (j + 1 < n_here) read(odd, s, j + 1);
            advance(even, j);
            if (j + 1 < n_here) {
                if (j + 2 < n_here) read(even, s, j + 2);
                advance(odd, j + 1);
            }
        }
        __syncthreads();                                     // the round's shares are there, its operands are done with
        for (int item = tid; item < n_here * DR_COLS; item += DR_THREADS) {
            const int j = item / DR_COLS, e = item % DR_COLS;
            float o = 0.f;
#pragma unroll
            for (int l = 0; l < DR_LANES; ++l) o += o_s[j][l][e];
            if (col0 + e < p.vdim) p.out[((size_t)(base + j) * p.heads + head) * p.vdim + col0 + e] = o;
        }
    }
#pragma unroll
    for (int u = 0; u < R4; ++u) {
        const int r = 4 * (lane + DR_LANES * u);
        if (live_col && r < p.dim) *reinterpret_cast<float4*>(s_base + r) = S[u];
    }
}

struct StepParams {
    DeltaParams d;
    const float* gate;          // rows gate_ld floats apart: [heads * vdim] logits
    const float* weight;        // [vdim]
    int gate_ld, out_ld, sigmoid_gate, true_vdim;
    float eps, out_scale;
};

// N sums over a warp that share their shuffles: on return lane l holds the sum number l / (32 / N)
template <int N>
__device__ __forceinline__ float shared_sums(float (&v)[N]) {
    const int lane = threadIdx.x & 31;
    int w = 16;
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
    for (; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
    return sum;
}

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
        const float sum_k = shared_sums<COLS>(held), sum_q = shared_sums<COLS>(seen);
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

template <int ROWS, int TOKENS, bool CHANNEL>
int launch_scan(const DeltaParams& p, int n_seqs, cudaStream_t stream) {
    constexpr size_t smem = 2 * sizeof(ScanStage<ROWS, TOKENS, CHANNEL>);
    static bool ready = false;
    if (!ready) {
        if (cudaFuncSetAttribute(delta_scan_kernel<ROWS, TOKENS, CHANNEL>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)smem) != cudaSuccess)
            MX_REFUSE("delta rule: cannot reserve %zu bytes of shared memory", smem);
        ready = true;
    }
    mx_launch_chained(delta_scan_kernel<ROWS, TOKENS, CHANNEL>, dim3(n_seqs, p.heads, (p.vdim + DR_COLS - 1) / DR_COLS),
                      dim3(DR_THREADS), smem, stream, p);
    return mx_launch_status();
}

template <bool CHANNEL>
int pick_scan(const DeltaParams& p, int n_seqs, cudaStream_t stream) {
    if (p.dim <= 32) return launch_scan<4, 16, CHANNEL>(p, n_seqs, stream);
    if (p.dim <= 64) return launch_scan<8, 16, CHANNEL>(p, n_seqs, stream);
    if (p.dim <= 128) return launch_scan<16, 16, CHANNEL>(p, n_seqs, stream);
    return launch_scan<32, 8, CHANNEL>(p, n_seqs, stream);
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
                        long long state_stride, long long state_offset, const int* cu_q, const int* state_slots, float* out,
                        int qk_heads, int heads, int dim, int vdim) {
    if (const char* what = delta_sizes(qk_heads, heads, dim, vdim)) MX_REFUSE("delta rule: %s: %d of %d, %d of %d", what, qk_heads, dim, heads, vdim);
    if (state_stride % 4 || state_offset % 4 || state_stride < state_offset + (long long)heads * dim * vdim)
        MX_REFUSE("delta rule: a state of %lld floats from %lld is too short", state_stride, state_offset);
    if (((uintptr_t)qkv | (uintptr_t)decay | (uintptr_t)state) % 16) MX_REFUSE("delta rule: unaligned operands");
    p.qkv = qkv; p.beta = beta; p.decay = decay; p.state = state; p.cu_q = cu_q; p.state_slots = state_slots; p.out = out;
    p.state_stride = state_stride; p.state_offset = state_offset; p.channels = 2 * qk_heads * dim + heads * vdim;
    p.k_col = qk_heads * dim; p.v_col = 2 * qk_heads * dim; p.qk_heads = qk_heads; p.heads = heads; p.dim = dim; p.vdim = vdim;
    return MX_OK;
}

// `per_channel`: decay is [tokens][heads][dim] instead of [tokens][heads]
extern "C" int mx_delta_scan(const float* qkv, const float* beta, const float* decay, int per_channel, float* state,
                             long long state_stride, long long state_offset, const int* cu_q, const int* state_slots,
                             float* out, int n_seqs, int qk_heads, int heads, int dim, int vdim, cudaStream_t stream) {
    if (n_seqs <= 0) return MX_OK;
    DeltaParams p;
    const int rc = delta_params(p, qkv, beta, decay, state, state_stride, state_offset, cu_q, state_slots, out, qk_heads, heads,
                                dim, vdim);
    if (rc != MX_OK) return rc;
    return per_channel ? pick_scan<true>(p, n_seqs, stream) : pick_scan<false>(p, n_seqs, stream);
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
    const int rc = delta_params(sp.d, qkv, beta, decay, state, state_stride, state_offset, cu_q, state_slots, nullptr, qk_heads,
                                heads, dim, vdim);
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
