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
