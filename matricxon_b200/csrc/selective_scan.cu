// A selective state-space recurrence (Mamba's) behind a short causal convolution.
//
// Per request the state is one float vector: the convolution's memory [taps - 1][channels] (conv_state.cuh), then the
// recurrent state [channels][n].
//
// mx_conv_silu: u_t = silu(conv(x)_t + conv_bias) per channel, from a column range of the input projection (float or
//   bfloat16 rows), written in the activation dtype. Memory rules as in conv_state.cuh.
// mx_selective_scan: every sequence's tokens in order, from and to its state:
//     dt = softplus(raw_t + dt_bias),  S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c u_c B_t[n],
//     out_t[c] = (sum_n S[c][n] C_t[n] + D_c u_c) * silu(z_t[c]) * out_scale
//   with A handed over as A * log2(e), so that the decay is one exp2. Everything but the operands u and z is float,
//   which are what the products and the convolution left (activation dtype).
//   A channel's states are shared out between LANES neighbouring threads, PER each, in registers for the whole
//   portion. Tokens arrive SCAN_TOKENS at a time through shared memory: while a round is computed, the next round's
//   operands are on their way into registers; steps, products and gates of a (token, channel) pair are formed once,
//   by the thread that stages it, and the lanes' shares of an output are added up once a round. The order of every
//   sum is fixed by this layout alone, so a token's result depends neither on the cut nor on the batch.
// mx_selective_scan_chunked: the same for long portions of few sequences, which the walk above leaves to a few warps per
//   SM. The recurrence is linear in S, and a chunk of tokens maps its start state to exp(A sum(dt)) S + (what the chunk
//   reaches from zero): the chunks' maps in parallel (all but a sequence's last), the start states chunk by chunk, then the
//   tokens of every chunk in parallel from its start state. Equal to the walk up to float rounding.
// mx_selective_step: the same for steps in which every sequence brings at most one token (decoding), with the product
//   that makes raw_t folded in: raw_t[c] = Wdt[c] . low_t, the low-rank row in float. The state sets out before the
//   wait on the kernel ahead.
#include <math.h>

#include "conv_state.cuh"

namespace {

constexpr int SCAN_THREADS = 128;
constexpr int SCAN_TOKENS = 16;

// ln(1 + e^x) for operands of type T: the library's functions for float, the hardware's exponential and logarithm for
// bfloat16 (a relative error of about 1e-5: where e^x is small, 1 + e^x has lost its digits and the series of ln(1 + e)
// takes over)
template <typename T> __device__ __forceinline__ float softplus_of(float x);
template <> __device__ __forceinline__ float softplus_of<float>(float x) { return x > 20.f ? x : log1pf(expf(x)); }
template <> __device__ __forceinline__ float softplus_of<__nv_bfloat16>(float x) {
    const float e = __expf(fminf(x, 20.f));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 1.f / 3.f), -0.5f), 1.f);
    const float y = e < 0.03125f ? series : fast_log2(1.f + e) * 0.6931471805599453f;
    return x > 20.f ? x : y;
}
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}

template <typename TIn, typename TOut>
__global__ void __launch_bounds__(256)
conv_silu_kernel(const TIn* x, int ld, const float* __restrict__ w, const float* __restrict__ bias, float* state,
                 long long state_stride, const int* __restrict__ tok_seq, const int* __restrict__ cu_q,
                 const int* __restrict__ state_slots, TOut* out, int channels, int taps) {
    pdl_trigger();
    const int t = blockIdx.x;
    const int seq = tok_seq[t];
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (seq < 0) {
        pdl_wait();
        if (c < channels) out[(size_t)t * channels + c] = from_float<TOut>(0.f);
        return;
    }
    const int first = cu_q[seq], local = t - first;
    const bool alone = cu_q[seq + 1] - first == 1;
    float* memory = state + (size_t)state_slots[seq] * state_stride;
    pdl_wait();
    if (c >= channels) return;
    const float y = conv_value(after_wait(x) + (size_t)first * ld, ld, memory, w, channels, taps, local, c, 0.f, alone);
    out[(size_t)t * channels + c] = from_float<TOut>(silu_of<TOut>(y + bias[c]));
}

// The same with a thread walking TOK neighbouring tokens of V channels, inputs in a window of registers.
template <typename TIn, typename TOut, int TAPS, int V, int TOK>
__global__ void __launch_bounds__(128)
conv_silu_window_kernel(const TIn* x, int ld, const float* __restrict__ w, const float* __restrict__ bias, float* state,
                        long long state_stride, const int* __restrict__ tok_seq, const int* __restrict__ cu_q,
                        const int* __restrict__ state_slots, TOut* out, int n_tokens, int channels) {
    pdl_trigger();
    const int t0 = blockIdx.x * TOK, c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= channels) return;
    ConvWindow<TAPS, V> window;
    window.weights(w, channels, c);
    const ConvVec<V> shift = conv_load<V>(bias + c);
    ConvVec<V> none;
#pragma unroll
    for (int e = 0; e < V; ++e) none.v[e] = 0.f;
    pdl_wait();
    x = after_wait(x);
    int seq_before = -1;
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        const int t = t0 + i;
        if (t >= n_tokens) break;
        const int seq = tok_seq[t];
        TOut* dst = out + (size_t)t * channels + c;
        if (seq < 0) {                                       // a padding row of a fixed-size batch
#pragma unroll
            for (int e = 0; e < V; ++e) dst[e] = from_float<TOut>(0.f);
            seq_before = -1;
            continue;
        }
        const int first = cu_q[seq];
        float* memory = state + (size_t)state_slots[seq] * state_stride;
        if (seq != seq_before) window.enter(x + (size_t)first * ld, ld, memory, channels, t - first, c, none);
        seq_before = seq;
        const ConvVec<V> y = window.step(conv_load<V>(x + (size_t)t * ld + c));
        if (cu_q[seq + 1] - first == 1) window.keep(memory, channels, c);
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = silu_of<TOut>(y.v[e] + shift.v[e]);
        if constexpr (V == 4 && sizeof(TOut) == 2) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(o[0], o[1]), hi = __floats2bfloat162_rn(o[2], o[3]);
            uint2 packed;
            packed.x = *reinterpret_cast<unsigned*>(&lo);
            packed.y = *reinterpret_cast<unsigned*>(&hi);
            *reinterpret_cast<uint2*>(dst) = packed;
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) dst[e] = from_float<TOut>(o[e]);
        }
    }
}

template <typename TIn, typename TOut, int TAPS>
void launch_conv_window(const TIn* x, int ld, const float* w, const float* bias, float* state, long long state_stride,
                        const int* tok_seq, const int* cu_q, const int* state_slots, TOut* out, int n_tokens, int channels,
                        cudaStream_t stream) {
    const int vecs = channels / 4, blocks = (vecs + 127) / 128;
    // few tokens: a block's walk would be the whole latency; many: neighbouring tokens share their inputs
    if (n_tokens <= 256)
        mx_launch_chained(conv_silu_window_kernel<TIn, TOut, TAPS, 4, 1>, dim3(n_tokens, blocks), dim3(128), 0, stream, x, ld,
                          w, bias, state, state_stride, tok_seq, cu_q, state_slots, out, n_tokens, channels);
    else
        mx_launch_chained(conv_silu_window_kernel<TIn, TOut, TAPS, 4, 8>, dim3((n_tokens + 7) / 8, blocks), dim3(128), 0,
                          stream, x, ld, w, bias, state, state_stride, tok_seq, cu_q, state_slots, out, n_tokens, channels);
}

struct ScanParams {
    const void* u;              // [tokens][channels], activation dtype
    const float* raw;           // scan: [tokens][raw_ld] before bias and softplus
    const float* low;           // [tokens][low_ld]: [dt_rank | B: n | C: n]
    const void* dt_weight;      // step: [channels][dt_rank], activation dtype
    const float* dt_bias;       // [channels]
    const float* a_log2;        // [channels][n]: A * log2(e), negative
    const float* d;             // [channels]
    const void* z;              // rows z_ld apart
    float* state;               // [slots][state_stride], the recurrent part at state_offset
    const int* cu_q;
    const int* state_slots;
    long long state_stride, state_offset;
    int raw_ld, low_ld, z_ld, out_ld, channels, n, dt_rank;
    float out_scale;
    // chunked form: [n_chunks][2] (sequence, first token of the chunk within its portion), [n_seqs + 1] first chunk of
    // every sequence; what a chunk reaches from zero and later its start state, and its sum of steps
    const int* chunks;
    const int* seq_chunk0;
    int chunk_tokens;
    float* chunk_state;         // [n_chunks][channels][n]
    float* chunk_dt;            // [n_chunks][channels]
};

// how a block of the scan kernel finds its tokens and its state
constexpr int SCAN_WHOLE = 0;   // a sequence's whole portion, from and to the state slot
constexpr int SCAN_MAPS = 1;    // a chunk from zero; its end and its sum of steps are kept, no outputs
constexpr int SCAN_TOKENS_OUT = 2;    // a chunk from its start state; the sequence's last one leaves the state

template <typename T, typename TZ, int PER, int LANES, int MODE>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_scan_kernel(const ScanParams p, T* __restrict__ out) {
    constexpr int CH = SCAN_THREADS / LANES;                 // channels per block
    constexpr int NP = PER * LANES;                          // states per channel, padded
    __shared__ __align__(16) float b_s[SCAN_TOKENS][NP], c_s[SCAN_TOKENS][NP];
    __shared__ __align__(8) float2 step_s[SCAN_TOKENS][CH];  // (dt, dt * u)
    __shared__ float y_s[SCAN_TOKENS][LANES][CH + 8];
    const int c0 = blockIdx.y * CH, tid = threadIdx.x;
    const int seq = MODE == SCAN_WHOLE ? (int)blockIdx.x : p.chunks[2 * blockIdx.x];
    int t0 = p.cu_q[seq], t1 = p.cu_q[seq + 1];
    if (t1 <= t0) return;
    bool last = true;
    if (MODE != SCAN_WHOLE) {
        last = (int)blockIdx.x == p.seq_chunk0[seq + 1] - 1;
        if (MODE == SCAN_MAPS && last) return;               // nobody asks what the last chunk hands on
        t0 += p.chunks[2 * blockIdx.x + 1];
        t1 = min(t1, t0 + p.chunk_tokens);
    }
    const int lane = tid % LANES, ch = tid / LANES, c = c0 + ch;
    float* kept = MODE == SCAN_WHOLE ? nullptr : p.chunk_state + ((size_t)blockIdx.x * p.channels + c) * p.n;
    float* s_row = p.state + (size_t)p.state_slots[seq] * p.state_stride + p.state_offset + (size_t)c * p.n;
    float S[PER], A[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int k = lane * PER + i;
        const bool live = c < p.channels && k < p.n;
        S[i] = live && MODE != SCAN_MAPS ? (MODE == SCAN_WHOLE ? s_row[k] : kept[k]) : 0.f;
        A[i] = live ? p.a_log2[(size_t)c * p.n + k] : 0.f;
    }
    float dt_sum = 0.f;
    constexpr int ITEMS = SCAN_TOKENS * CH / SCAN_THREADS;   // (token, channel) pairs a thread stages
    constexpr int BC_ITEMS = (SCAN_TOKENS * NP + SCAN_THREADS - 1) / SCAN_THREADS;
    static_assert(SCAN_TOKENS * CH % SCAN_THREADS == 0, "every thread stages the same number of pairs");
    float raw_r[ITEMS], u_r[ITEMS], z_r[ITEMS], b_r[BC_ITEMS], c_r[BC_ITEMS];
    const T* u = reinterpret_cast<const T*>(p.u);
    const TZ* z = reinterpret_cast<const TZ*>(p.z);
    auto fetch = [&](int base) {
        const int here = min(SCAN_TOKENS, t1 - base);
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int item = tid + i * SCAN_THREADS, j = item / CH, cc = c0 + item % CH;
            const bool live = j < here && cc < p.channels;
            const size_t t = (size_t)(base + j);
            raw_r[i] = live ? p.raw[t * p.raw_ld + cc] : 0.f;
            u_r[i] = live ? to_float(u[t * p.channels + cc]) : 0.f;
            if (MODE != SCAN_MAPS) z_r[i] = live ? to_float(z[t * p.z_ld + cc]) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < BC_ITEMS; ++i) {
            const int item = tid + i * SCAN_THREADS, j = item / NP, k = item % NP;
            const bool live = j < here && k < p.n;
            const float* row = p.low + (size_t)(base + j) * p.low_ld + p.dt_rank;
            b_r[i] = live ? row[k] : 0.f;
            if (MODE != SCAN_MAPS) c_r[i] = live ? row[p.n + k] : 0.f;
        }
    };
    float skip[ITEMS], gate[ITEMS];
    float dt_bias[ITEMS], d_skip[ITEMS];                     // constants of the pairs this thread stages
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
        const int cc = c0 + (tid + i * SCAN_THREADS) % CH;
        dt_bias[i] = cc < p.channels ? p.dt_bias[cc] : 0.f;
        d_skip[i] = cc < p.channels ? p.d[cc] : 0.f;
    }
    fetch(t0);
    for (int base = t0; base < t1; base += SCAN_TOKENS) {
        const int here = min(SCAN_TOKENS, t1 - base);
        __syncthreads();
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int item = tid + i * SCAN_THREADS, j = item / CH, k = item % CH;
            const float dt = softplus_of<T>(raw_r[i] + dt_bias[i]);
            step_s[j][k] = make_float2(dt, dt * u_r[i]);
            // this thread writes the pair's output as well: its skip term and gate stay in registers
            if (MODE != SCAN_MAPS) {
                skip[i] = d_skip[i] * u_r[i];
                gate[i] = silu_of<T>(z_r[i]) * p.out_scale;
            }
        }
#pragma unroll
        for (int i = 0; i < BC_ITEMS; ++i) {
            const int item = tid + i * SCAN_THREADS;
            if (item < SCAN_TOKENS * NP) {
                b_s[item / NP][item % NP] = b_r[i];
                if (MODE != SCAN_MAPS) c_s[item / NP][item % NP] = c_r[i];
            }
        }
        __syncthreads();
        if (base + SCAN_TOKENS < t1) fetch(base + SCAN_TOKENS);
#pragma unroll 4
        for (int j = 0; j < here; ++j) {
            const float2 step = step_s[j][ch];
            float y = 0.f;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                S[i] = fmaf(exp2_fast(step.x * A[i]), S[i], step.y * b_s[j][lane * PER + i]);
                if (MODE != SCAN_MAPS) y = fmaf(S[i], c_s[j][lane * PER + i], y);
            }
            if (MODE == SCAN_MAPS) dt_sum += step.x;
            else y_s[j][lane][ch] = y;
        }
        if (MODE == SCAN_MAPS) continue;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int item = tid + i * SCAN_THREADS, j = item / CH, k = item % CH;
            if (j < here && c0 + k < p.channels) {
                float y = skip[i];
#pragma unroll
                for (int l = 0; l < LANES; ++l) y += y_s[j][l][k];
                out[(size_t)(base + j) * p.out_ld + c0 + k] = from_float<T>(y * gate[i]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int k = lane * PER + i;
        if (c < p.channels && k < p.n) {
            if (MODE == SCAN_MAPS) kept[k] = S[i];
            else if (last) s_row[k] = S[i];
        }
    }
    if (MODE == SCAN_MAPS && lane == 0 && c < p.channels) p.chunk_dt[(size_t)blockIdx.x * p.channels + c] = dt_sum;
}

// The chunks' start states in order, in place of what they reach from zero: a thread per (sequence, channel, state).
__global__ void __launch_bounds__(256)
selective_carry_kernel(const ScanParams p) {
    const int seq = blockIdx.x;
    const long long i = (long long)blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= (long long)p.channels * p.n || p.cu_q[seq + 1] <= p.cu_q[seq]) return;
    const int c = (int)(i / p.n);
    const float a = p.a_log2[i];
    float s = p.state[(size_t)p.state_slots[seq] * p.state_stride + p.state_offset + i];
    const int end = p.seq_chunk0[seq + 1];
    const size_t stride = (size_t)p.channels * p.n;
    constexpr int AHEAD = 8;                                 // a group's maps are read before its first start is written
    for (int chunk = p.seq_chunk0[seq]; chunk < end; chunk += AHEAD) {
        float* here = p.chunk_state + (size_t)chunk * stride + i;
        const float* dt = p.chunk_dt + (size_t)chunk * p.channels + c;
        float reached[AHEAD], passed[AHEAD];
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
            const bool maps = chunk + g + 1 < end;           // the last chunk hands nothing on
            reached[g] = maps ? here[g * stride] : 0.f;
            passed[g] = maps ? dt[(size_t)g * p.channels] : 0.f;
        }
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
            if (chunk + g >= end) break;
            here[g * stride] = s;
            s = fmaf(exp2_fast(passed[g] * a), s, reached[g]);
        }
    }
}

template <typename T, typename TZ, int PER, int LANES>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_step_kernel(const ScanParams p, T* out) {
    constexpr int CH = SCAN_THREADS / LANES;
    pdl_trigger();
    const int seq = blockIdx.x, tid = threadIdx.x;
    const int t = p.cu_q[seq];
    const int lane = tid % LANES, c = blockIdx.y * CH + tid / LANES;
    if (p.cu_q[seq + 1] <= t) {
        // a padding sequence of a fixed-size batch, whose row bears its own number: defined output, no state
        pdl_wait();
        if (seq >= t && lane == 0 && c < p.channels) out[(size_t)seq * p.out_ld + c] = from_float<T>(0.f);
        return;
    }
    const bool mine = c < p.channels;
    const int cc = mine ? c : p.channels - 1;                // idle channels compute the last one and store nothing
    float* s_row = p.state + (size_t)p.state_slots[seq] * p.state_stride + p.state_offset + (size_t)cc * p.n;
    float S[PER], A[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {                          // the state of earlier steps and constants of the layer
        const int k = lane * PER + i;
        S[i] = k < p.n ? s_row[k] : 0.f;
        A[i] = k < p.n ? p.a_log2[(size_t)cc * p.n + k] : 0.f;
    }
    const float dt_bias = p.dt_bias[cc], d_skip = p.d[cc];
    const T* w = reinterpret_cast<const T*>(p.dt_weight) + (size_t)cc * p.dt_rank;
    prefetch_l2(w + min(lane * ((p.dt_rank + LANES - 1) / LANES), p.dt_rank - 1));
    pdl_wait();
    const float* low = after_wait(p.low) + (size_t)t * p.low_ld;
    float raw = 0.f;
    if (p.dt_rank % 4 == 0 && p.low_ld % 4 == 0) {
        // a thread takes every LANES-th group of four entries of the row
        for (int r = 4 * lane; r < p.dt_rank; r += 4 * LANES) {
            const float4 l = *reinterpret_cast<const float4*>(low + r);
            raw = fmaf(to_float(w[r]), l.x, raw);
            raw = fmaf(to_float(w[r + 1]), l.y, raw);
            raw = fmaf(to_float(w[r + 2]), l.z, raw);
            raw = fmaf(to_float(w[r + 3]), l.w, raw);
        }
    } else {
        for (int r = lane; r < p.dt_rank; r += LANES) raw = fmaf(to_float(w[r]), low[r], raw);
    }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) raw += __shfl_xor_sync(0xffffffffu, raw, o);
    const float u = to_float(reinterpret_cast<const T*>(after_wait(p.u))[(size_t)t * p.channels + cc]);
    const float z = to_float(reinterpret_cast<const TZ*>(after_wait(p.z))[(size_t)t * p.z_ld + cc]);
    const float dt = softplus_of<T>(raw + dt_bias), du = dt * u;
    const float* b = low + p.dt_rank;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int k = lane * PER + i;
        if (k < p.n) {
            S[i] = fmaf(exp2_fast(dt * A[i]), S[i], du * b[k]);
            y = fmaf(S[i], b[p.n + k], y);
            if (mine) s_row[k] = S[i];
        }
    }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (mine && lane == 0) out[(size_t)t * p.out_ld + c] = from_float<T>((y + d_skip * u) * silu_of<T>(z) * p.out_scale);
}

template <typename T, typename TZ>
int launch_scan(const ScanParams& p, T* out, int n_seqs, int n_chunks, bool step, cudaStream_t stream) {
#define MX_SCAN(PER, LANES)                                                                                            \
    do {                                                                                                               \
        const int tiles = (p.channels + SCAN_THREADS / LANES - 1) / (SCAN_THREADS / LANES);                           \
        const dim3 grid(n_chunks > 0 ? n_chunks : n_seqs, tiles);                                                      \
        if (n_chunks > 0) {                                                                                            \
            selective_scan_kernel<T, TZ, PER, LANES, SCAN_MAPS><<<grid, SCAN_THREADS, 0, stream>>>(p, out);            \
            const long long states = (long long)p.channels * p.n;                                                      \
            selective_carry_kernel<<<dim3(n_seqs, (unsigned)((states + 255) / 256)), 256, 0, stream>>>(p);             \
            selective_scan_kernel<T, TZ, PER, LANES, SCAN_TOKENS_OUT><<<grid, SCAN_THREADS, 0, stream>>>(p, out);      \
        } else if (step)                                                                                                      \
            mx_launch_chained(selective_step_kernel<T, TZ, PER, LANES>, grid, dim3(SCAN_THREADS), 0, stream, p, out); \
        else                                                                                                           \
            selective_scan_kernel<T, TZ, PER, LANES, SCAN_WHOLE><<<grid, SCAN_THREADS, 0, stream>>>(p, out);          \
        return mx_launch_status();                                                                                     \
    } while (0)
    const int n = p.n;
    if (n <= 4) MX_SCAN(1, 4);
    if (n <= 8) MX_SCAN(2, 4);
    if (n <= 16) MX_SCAN(4, 4);
    if (n <= 24) MX_SCAN(6, 4);
    if (n <= 32) MX_SCAN(8, 4);
    if (n <= 64) MX_SCAN(16, 4);
    MX_SCAN(8, 16);
#undef MX_SCAN
}

int run_scan(const ScanParams& p, void* out, int dtype, int z_dtype, int n_seqs, int n_chunks, bool step,
             cudaStream_t stream) {
    if (n_seqs <= 0 || p.channels <= 0) return MX_OK;
    if (p.n <= 0 || p.n > 128) MX_REFUSE("selective scan: %d states per channel (1..128)", p.n);
    if (p.dt_rank <= 0) MX_REFUSE("selective scan: a step rank of %d", p.dt_rank);
    if (p.low_ld < p.dt_rank + 2 * p.n) MX_REFUSE("selective scan: rows of %d hold no [%d | %d | %d]", p.low_ld, p.dt_rank, p.n, p.n);
    if (p.channels > 65535 * 8) MX_REFUSE("selective scan: %d channels exceed the grid", p.channels);
    if (p.state_stride < p.state_offset + (long long)p.channels * p.n) MX_REFUSE("selective scan: a state of %lld floats is too short", p.state_stride);
    if (dtype == MX_DTYPE_F32) {
        if (z_dtype != MX_DTYPE_F32) MX_REFUSE("selective scan: a bfloat16 gate beside float activations");
        return launch_scan<float, float>(p, (float*)out, n_seqs, n_chunks, step, stream);
    }
    if (z_dtype == MX_DTYPE_F32)
        return launch_scan<__nv_bfloat16, float>(p, (__nv_bfloat16*)out, n_seqs, n_chunks, step, stream);
    return launch_scan<__nv_bfloat16, __nv_bfloat16>(p, (__nv_bfloat16*)out, n_seqs, n_chunks, step, stream);
}

}  // namespace

extern "C" int mx_conv_silu(const void* x, int in_dtype, int ld, const float* w, const float* bias, float* state,
                            long long state_stride, const int* tok_seq, const int* cu_q, const int* state_slots, void* out,
                            int out_dtype, int n_tokens, int channels, int taps, cudaStream_t stream) {
    if (n_tokens <= 0 || channels <= 0) return MX_OK;
    if (taps < 1) MX_REFUSE("convolution: %d taps", taps);
    if (state_stride < (long long)(taps - 1) * channels) MX_REFUSE("convolution: a state of %lld floats is too short", state_stride);
    // the windowed form reads 4 channels at once: aligned columns, strides and state rows
    const bool vec = channels % 4 == 0 && ld % 4 == 0 && state_stride % 4 == 0 && (uintptr_t)x % (in_dtype == MX_DTYPE_F32 ? 16 : 8) == 0 &&
                     ((uintptr_t)w | (uintptr_t)bias | (uintptr_t)state | (uintptr_t)out) % 16 == 0;
    const dim3 grid(n_tokens, (channels + 255) / 256);
#define MX_CONV_WINDOW(TI, TO, TAPS)                                                                                \
    launch_conv_window<TI, TO, TAPS>((const TI*)x, ld, w, bias, state, state_stride, tok_seq, cu_q, state_slots,    \
                                     (TO*)out, n_tokens, channels, stream)
#define MX_CONV(TI, TO)                                                                                             \
    if (vec && taps == 2) MX_CONV_WINDOW(TI, TO, 2);                                                                \
    else if (vec && taps == 3) MX_CONV_WINDOW(TI, TO, 3);                                                           \
    else if (vec && taps == 4) MX_CONV_WINDOW(TI, TO, 4);                                                           \
    else                                                                                                            \
    mx_launch_chained(conv_silu_kernel<TI, TO>, grid, dim3(256), 0, stream, (const TI*)x, ld, w, bias, state,      \
                      state_stride, tok_seq, cu_q, state_slots, (TO*)out, channels, taps)
    if (in_dtype == MX_DTYPE_F32 && out_dtype == MX_DTYPE_F32) { MX_CONV(float, float); }
    else if (in_dtype == MX_DTYPE_F32) { MX_CONV(float, __nv_bfloat16); }
    else if (out_dtype == MX_DTYPE_BF16) { MX_CONV(__nv_bfloat16, __nv_bfloat16); }
    else MX_REFUSE("convolution: bfloat16 inputs with a float output are not used by any path");
#undef MX_CONV
#undef MX_CONV_WINDOW
    return mx_launch_status();
}

extern "C" int mx_selective_scan(const void* u, const float* raw, int raw_ld, const float* low, int low_ld,
                                 const float* dt_bias, const float* a_log2, const float* d, const void* z, int z_dtype,
                                 int z_ld, float* state, long long state_stride, long long state_offset, const int* cu_q,
                                 const int* state_slots, void* out, int dtype, int out_ld, int n_seqs, int channels, int n,
                                 int dt_rank, float out_scale, cudaStream_t stream) {
    const ScanParams p = {u, raw, low, nullptr, dt_bias, a_log2, d, z, state, cu_q, state_slots, state_stride, state_offset,
                          raw_ld, low_ld, z_ld, out_ld, channels, n, dt_rank, out_scale, nullptr, nullptr, 0, nullptr, nullptr};
    return run_scan(p, out, dtype, z_dtype, n_seqs, 0, false, stream);
}

// `chunks` [n_chunks][2] (sequence, first token within its portion), sequence by sequence in chunks of `chunk_tokens`
// tokens; `seq_chunk0` [n_seqs + 1]; `scratch` n_chunks * channels * (n + 1) floats.
extern "C" int mx_selective_scan_chunked(const void* u, const float* raw, int raw_ld, const float* low, int low_ld,
                                         const float* dt_bias, const float* a_log2, const float* d, const void* z, int z_dtype,
                                         int z_ld, float* state, long long state_stride, long long state_offset,
                                         const int* cu_q, const int* state_slots, void* out, int dtype, int out_ld, int n_seqs,
                                         int channels, int n, int dt_rank, float out_scale, const int* chunks,
                                         const int* seq_chunk0, int n_chunks, int chunk_tokens, float* scratch,
                                         cudaStream_t stream) {
    if (n_chunks <= 0) return MX_OK;
    if (chunk_tokens <= 0) MX_REFUSE("selective scan: chunks of %d tokens", chunk_tokens);
    const ScanParams p = {u, raw, low, nullptr, dt_bias, a_log2, d, z, state, cu_q, state_slots, state_stride, state_offset,
                          raw_ld, low_ld, z_ld, out_ld, channels, n, dt_rank, out_scale, chunks, seq_chunk0, chunk_tokens,
                          scratch, scratch + (size_t)n_chunks * channels * n};
    return run_scan(p, out, dtype, z_dtype, n_seqs, n_chunks, false, stream);
}

extern "C" int mx_selective_step(const void* u, const float* low, int low_ld, const void* dt_weight, const float* dt_bias,
                                 const float* a_log2, const float* d, const void* z, int z_dtype, int z_ld, float* state,
                                 long long state_stride, long long state_offset, const int* cu_q, const int* state_slots,
                                 void* out, int dtype, int out_ld, int n_seqs, int channels, int n, int dt_rank,
                                 float out_scale, cudaStream_t stream) {
    const ScanParams p = {u, nullptr, low, dt_weight, dt_bias, a_log2, d, z, state, cu_q, state_slots, state_stride,
                          state_offset, 0, low_ld, z_ld, out_ld, channels, n, dt_rank, out_scale, nullptr, nullptr, 0, nullptr,
                          nullptr};
    return run_scan(p, out, dtype, z_dtype, n_seqs, 0, true, stream);
}
