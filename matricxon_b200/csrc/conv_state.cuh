// Short causal convolutions over a flattened batch of sequence portions, with the latest inputs kept per request.
//
// A request's memory of a convolution with `taps` taps over C channels is a float matrix [taps - 1][C] (oldest input
// first) at the start of its state vector; a new request's is zero, which is what the convolution reads before a
// sequence's start. The kernels that convolve read the memory for the first taps - 1 tokens of a portion. A sequence
// that brings one token has its memory moved on by the thread that convolves it (nobody else reads that channel); one
// that brings more has it rewritten by mx_conv_state_update afterwards, since other blocks still read the old one.
#pragma once

#include "common.cuh"

// The input of channel `c` `back` tokens before the local token `local` of a portion whose first row is `first_row`
// (row pointer of column 0 of the convolved columns, rows `ld` apart). Inputs carry `bias` except the kept ones,
// which were stored with it.
template <typename T>
__device__ __forceinline__ float conv_input(const T* first_row, int ld, const float* memory, int channels, int taps,
                                            int local, int back, int c, float bias) {
    return local >= back ? to_float(first_row[(size_t)(local - back) * ld + c]) + bias
                         : memory[(size_t)(taps - 1 + local - back) * channels + c];
}

// The inputs of V neighbouring channels from c on (a multiple of V), one 16-byte access where V is 4.
template <int V> struct ConvVec { float v[V]; };
template <int V, typename T>
__device__ __forceinline__ ConvVec<V> conv_load(const T* p) {
    ConvVec<V> r;
    if constexpr (V == 4 && sizeof(T) == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    } else if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        r.v[0] = __uint_as_float(raw.x << 16); r.v[1] = __uint_as_float(raw.x & 0xffff0000u);
        r.v[2] = __uint_as_float(raw.y << 16); r.v[3] = __uint_as_float(raw.y & 0xffff0000u);
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = to_float(p[e]);
    }
    return r;
}
template <int V>
__device__ __forceinline__ void conv_store(float* p, const ConvVec<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else {
#pragma unroll
        for (int e = 0; e < V; ++e) p[e] = r.v[e];
    }
}

// A thread's walk over neighbouring tokens with the TAPS - 1 inputs before the current one in registers (oldest first).
// `enter` fills them for the token `local` of a sequence; `step` takes the token's own input, gives the convolution's
// value and moves on; `keep` leaves them as the sequence's memory (for a portion of one token, right behind its step).
template <int TAPS, int V>
struct ConvWindow {
    ConvVec<V> past[TAPS > 1 ? TAPS - 1 : 1], w[TAPS];

    __device__ __forceinline__ void weights(const float* conv, int channels, int c) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = conv_load<V>(conv + (size_t)j * channels + c);
    }
    template <typename T>
    __device__ __forceinline__ void enter(const T* first_row, int ld, const float* memory, int channels, int local, int c,
                                          const ConvVec<V>& bias) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int back = TAPS - 1 - j;
            if (local >= back) {
                past[j] = conv_load<V>(first_row + (size_t)(local - back) * ld + c);
#pragma unroll
                for (int e = 0; e < V; ++e) past[j].v[e] += bias.v[e];
            } else {
                past[j] = conv_load<V>(memory + (size_t)(TAPS - 1 + local - back) * channels + c);
            }
        }
    }
    __device__ __forceinline__ ConvVec<V> step(const ConvVec<V>& u) {
        ConvVec<V> y;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) sum = fmaf(w[j].v[e], past[j].v[e], sum);
            y.v[e] = fmaf(w[TAPS - 1].v[e], u.v[e], sum);
        }
#pragma unroll
        for (int j = 0; j + 1 < TAPS - 1; ++j) past[j] = past[j + 1];
        if (TAPS > 1) past[TAPS > 1 ? TAPS - 2 : 0] = u;
        return y;
    }
    __device__ __forceinline__ void keep(float* memory, int channels, int c) const {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) conv_store<V>(memory + (size_t)j * channels + c, past[j]);
    }
};

// sum_j w[j][c] * input (taps - 1 - j) tokens back; w is [taps][C]. With `move_on` (the portion is this one token)
// the channel's memory is shifted by the token's own input.
template <typename T>
__device__ __forceinline__ float conv_value(const T* first_row, int ld, float* memory, const float* w, int channels,
                                            int taps, int local, int c, float bias, bool move_on) {
    float y = 0.f;
    for (int j = 0; j < taps; ++j) {
        const float u = conv_input(first_row, ld, memory, channels, taps, local, taps - 1 - j, c, bias);
        y = fmaf(w[(size_t)j * channels + c], u, y);
        if (move_on && j > 0) memory[(size_t)(j - 1) * channels + c] = u;      // input j - 1 of the next token
    }
    return y;
}
