// The step ahead of an attention whose projections pass a short causal convolution and whose queries and keys are
// RMS-normalised over the whole projection (all heads at once).
//
// mx_conv_norm_kv_write: float rows [q heads x dim | k heads x dim | v heads x vdim] of a fused projection (k and v
//   absent where the layer attends over another layer's cache: n_kv_heads is then only the geometry of that cache)
//   become the operands of the paged attention kernels. For every channel u = proj + bias,
//   y_t = sum_j w[j] u_(t - taps + 1 + j) with the portion's earlier inputs from the request's memory (conv_state.cuh);
//     q_out [tokens][heads * hd]                 unit(y over all q channels) * q_weight * temperature(position)
//     cache keys   [page][0][kv head][slot][hd]  unit(y over all k channels) * k_weight
//     cache values [page][1][kv head][hd][slot]  y
//   heads padded with zeros from dim (vdim) to hd. unit(x) = x / sqrt(mean(x^2) + eps);
//   temperature(p) = 1 + coef * ln(floor((p + 1) / every) + 1). All of it is float; results are rounded once.
//   A block owns a token (any sizes and taps) or, for two to four taps and widths in groups of four, one or four
//   neighbouring tokens with 16-byte accesses; the convolved rows lie in shared memory between the passes.
// mx_conv_state_update: the memory of sequences that bring two or more tokens, after everybody has read it.
#include <math.h>

#include "conv_state.cuh"

namespace {

struct ConvAttnParams {
    const float* proj;          // [tokens][ld]
    const float* bias;          // [C] or null
    const float* conv;          // [taps][C]
    const float* q_weight;      // [heads * dim]
    const float* k_weight;      // [kv heads * dim]
    float* state;               // [slots][state_stride], memory [taps - 1][C] first
    const int* positions;
    const int* tok_seq;
    const int* cu_q;
    const int* state_slots;
    const int* slots;           // null: nothing is stored
    int* status;
    long long n_slots, state_stride;
    int ld, taps, n_heads, n_kv_heads, dim, vdim, hd, page_size, own_kv;
    float eps, temp_coef, temp_every;
};

template <typename T>
__global__ void __launch_bounds__(256)
conv_norm_kv_write_kernel(const ConvAttnParams p, T* __restrict__ cache, T* __restrict__ q_out) {
    extern __shared__ float row[];                            // [C] convolved values
    __shared__ float scratch[32];
    pdl_trigger();
    const int t = blockIdx.x, tid = threadIdx.x;
    const int q_width = p.n_heads * p.dim, k_width = p.own_kv ? p.n_kv_heads * p.dim : 0;
    const int v_width = p.own_kv ? p.n_kv_heads * p.vdim : 0;
    const int channels = q_width + k_width + v_width;
    T* q_row = q_out + (size_t)t * p.n_heads * p.hd;
    const int seq = p.tok_seq[t];
    if (seq < 0) {                                            // a padding row of a fixed-size batch
        pdl_wait();
        for (int i = tid; i < p.n_heads * p.hd; i += blockDim.x) q_row[i] = from_float<T>(0.f);
        return;
    }
    const int first = p.cu_q[seq], local = t - first;
    const bool alone = p.cu_q[seq + 1] - first == 1;
    const float pos = (float)p.positions[t];
    const float temperature = 1.f + p.temp_coef * logf(floorf(__fdiv_rn(pos + 1.f, p.temp_every)) + 1.f);
    float* memory = p.state + (size_t)p.state_slots[seq] * p.state_stride;
    long long slot = p.own_kv && p.slots ? p.slots[t] : -1;
    if (slot != -1 && (slot < 0 || slot >= p.n_slots)) {
        if (tid == 0) atomicOr(p.status, MX_STATUS_BAD_SLOT);
        slot = -1;
    }
    pdl_wait();
    const float* first_row = after_wait(p.proj) + (size_t)first * p.ld;
    float q_sum = 0.f, k_sum = 0.f;
    for (int c = tid; c < channels; c += blockDim.x) {
        const float y = conv_value(first_row, p.ld, memory, p.conv, channels, p.taps, local, c, p.bias ? p.bias[c] : 0.f,
                                   alone);
        row[c] = y;
        if (c < q_width) q_sum = fmaf(y, y, q_sum);
        else if (c < q_width + k_width) k_sum = fmaf(y, y, k_sum);
    }
    const float q_inv = temperature / sqrtf(block_sum(q_sum, scratch) / (float)q_width + p.eps);
    for (int i = tid; i < p.n_heads * p.hd; i += blockDim.x) {
        const int h = i / p.hd, d = i - h * p.hd, c = h * p.dim + d;
        q_row[i] = from_float<T>(d < p.dim ? row[c] * q_inv * p.q_weight[c] : 0.f);
    }
    if (!p.own_kv) return;
    const float k_inv = 1.f / sqrtf(block_sum(k_sum, scratch) / (float)k_width + p.eps);
    if (slot < 0) return;
    const long long page = slot / p.page_size;
    const int offset = (int)(slot - page * p.page_size);
    const size_t head_stride = (size_t)p.page_size * p.hd;
    T* kbase = cache + ((size_t)page * 2 * p.n_kv_heads) * head_stride + (size_t)offset * p.hd;
    T* vbase = cache + ((size_t)page * 2 * p.n_kv_heads + p.n_kv_heads) * head_stride + offset;
    for (int i = tid; i < p.n_kv_heads * p.hd; i += blockDim.x) {
        const int h = i / p.hd, d = i - h * p.hd;
        const int kc = h * p.dim + d, vc = h * p.vdim + d;
        kbase[(size_t)h * head_stride + d] = from_float<T>(d < p.dim ? row[q_width + kc] * k_inv * p.k_weight[kc] : 0.f);
        vbase[(size_t)h * head_stride + (size_t)d * p.page_size] =
            from_float<T>(d < p.vdim ? row[q_width + k_width + vc] : 0.f);
    }
}

// TOK neighbouring tokens per block: a thread owns V neighbouring channels of all of them (inputs in a window of
// registers, the convolution's weights read once), the convolved rows lie in shared memory between the passes.
template <typename T, int TAPS, int V, int TOK>
__global__ void __launch_bounds__(512)
conv_norm_window_kernel(const ConvAttnParams p, T* __restrict__ cache, T* __restrict__ q_out, int n_tokens) {
    extern __shared__ __align__(16) float rows[];             // [TOK][channels]
    __shared__ float partial[2][TOK][16];                     // per warp: sums of squares of q and of k
    __shared__ float inv[2][TOK];
    pdl_trigger();
    const int t0 = blockIdx.x * TOK, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int here = min(TOK, n_tokens - t0);
    const int q_width = p.n_heads * p.dim, k_width = p.own_kv ? p.n_kv_heads * p.dim : 0;
    const int v_width = p.own_kv ? p.n_kv_heads * p.vdim : 0;
    const int channels = q_width + k_width + v_width;
    float q_sum[TOK], k_sum[TOK];
#pragma unroll
    for (int i = 0; i < TOK; ++i) q_sum[i] = k_sum[i] = 0.f;
    pdl_wait();
    const float* proj = after_wait(p.proj);
    for (int c = tid * V; c < channels; c += blockDim.x * V) {
        ConvWindow<TAPS, V> window;
        window.weights(p.conv, channels, c);
        ConvVec<V> bias;
        if (p.bias) bias = conv_load<V>(p.bias + c);
        else {
#pragma unroll
            for (int e = 0; e < V; ++e) bias.v[e] = 0.f;
        }
        ConvVec<V> own[TOK];                                  // every token's own inputs set out together
#pragma unroll
        for (int i = 0; i < TOK; ++i)
            if (i < here) own[i] = conv_load<V>(proj + (size_t)(t0 + i) * p.ld + c);
        int seq_before = -1;
#pragma unroll
        for (int i = 0; i < TOK; ++i) {
            if (i >= here) break;
            const int t = t0 + i, seq = p.tok_seq[t];
            if (seq < 0) {                                    // a padding row of a fixed-size batch
                seq_before = -1;
                continue;
            }
            const int first = p.cu_q[seq];
            float* memory = p.state + (size_t)p.state_slots[seq] * p.state_stride;
            if (seq != seq_before)
                window.enter(proj + (size_t)first * p.ld, p.ld, memory, channels, t - first, c, bias);
            seq_before = seq;
            ConvVec<V> u = own[i];
#pragma unroll
            for (int e = 0; e < V; ++e) u.v[e] += bias.v[e];
            const ConvVec<V> y = window.step(u);
            if (p.cu_q[seq + 1] - first == 1) window.keep(memory, channels, c);
            conv_store<V>(rows + (size_t)i * channels + c, y);
            float s = 0.f;
#pragma unroll
            for (int e = 0; e < V; ++e) s = fmaf(y.v[e], y.v[e], s);
            if (c < q_width) q_sum[i] += s;                   // V divides the widths: a group lies in one part
            else if (c < q_width + k_width) k_sum[i] += s;
        }
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        const float q = warp_sum(q_sum[i]), k = warp_sum(k_sum[i]);
        if (lane == 0) { partial[0][i][warp] = q; partial[1][i][warp] = k; }
    }
    __syncthreads();
    if (tid < 2 * TOK) {
        const int part = tid & 1, i = tid >> 1;
        float s = 0.f;
        for (int w = 0; w < (int)(blockDim.x >> 5); ++w) s += partial[part][i][w];
        const int width = part ? k_width : q_width;
        float r = width > 0 ? 1.f / sqrtf(s / (float)width + p.eps) : 0.f;
        if (part == 0 && i < here) {
            const float pos = (float)p.positions[t0 + i];
            r *= 1.f + p.temp_coef * logf(floorf(__fdiv_rn(pos + 1.f, p.temp_every)) + 1.f);
        }
        inv[part][i] = r;
    }
    __syncthreads();
    const int hd4 = p.hd / 4;                                 // heads are padded to a multiple of 16
    auto put4 = [](T* dst, float a, float b, float c, float d) {
        if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
        else {
            __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
            uint2 packed;
            packed.x = *reinterpret_cast<unsigned*>(&lo);
            packed.y = *reinterpret_cast<unsigned*>(&hi);
            *reinterpret_cast<uint2*>(dst) = packed;
        }
    };
    // four entries of a head (zeros behind its `dim`), normalised
    auto head4 = [&](const float* row, const float* weight, int h, int d, float scale, float* o) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = h * p.dim + d + e;
            o[e] = d + e < p.dim ? row[c] * scale * weight[c] : 0.f;
        }
    };
    for (int i = 0; i < here; ++i) {
        const int t = t0 + i, seq = p.tok_seq[t];
        const float* row = rows + (size_t)i * channels;
        T* q_row = q_out + (size_t)t * p.n_heads * p.hd;
        for (int item = tid; item < p.n_heads * hd4; item += blockDim.x) {
            const int h = item / hd4, d = (item - h * hd4) * 4;
            float o[4] = {0.f, 0.f, 0.f, 0.f};
            if (seq >= 0) head4(row, p.q_weight, h, d, inv[0][i], o);
            put4(q_row + (size_t)h * p.hd + d, o[0], o[1], o[2], o[3]);
        }
        if (!p.own_kv || seq < 0 || p.slots == nullptr) continue;
        const long long slot = p.slots[t];
        if (slot == -1) continue;
        if (slot < 0 || slot >= p.n_slots) {
            if (tid == 0) atomicOr(p.status, MX_STATUS_BAD_SLOT);
            continue;
        }
        const long long page = slot / p.page_size;
        const int offset = (int)(slot - page * p.page_size);
        const size_t head_stride = (size_t)p.page_size * p.hd;
        T* kbase = cache + ((size_t)page * 2 * p.n_kv_heads) * head_stride + (size_t)offset * p.hd;
        T* vbase = cache + ((size_t)page * 2 * p.n_kv_heads + p.n_kv_heads) * head_stride + offset;
        for (int item = tid; item < p.n_kv_heads * hd4; item += blockDim.x) {
            const int h = item / hd4, d = (item - h * hd4) * 4;
            float o[4];
            head4(row + q_width, p.k_weight, h, d, inv[1][i], o);
            put4(kbase + (size_t)h * head_stride + d, o[0], o[1], o[2], o[3]);
        }
        for (int item = tid; item < p.n_kv_heads * p.hd; item += blockDim.x) {
            const int h = item / p.hd, d = item - h * p.hd;
            vbase[(size_t)h * head_stride + (size_t)d * p.page_size] =
                from_float<T>(d < p.vdim ? row[q_width + k_width + h * p.vdim + d] : 0.f);
        }
    }
}

template <typename T, int TAPS>
int launch_window(const ConvAttnParams& p, T* cache, T* q_out, int n_tokens, int channels, cudaStream_t stream) {
    // few tokens: a token's latency is all there is; many: neighbours share inputs and weights
    constexpr int TOK = 4;
    const bool many = n_tokens > 256 && (size_t)channels * TOK * sizeof(float) <= 100 * 1024;
    const size_t smem = (size_t)channels * (many ? TOK : 1) * sizeof(float);
    const int vecs = (channels + 3) / 4;
    if (many) {
        auto kernel = conv_norm_window_kernel<T, TAPS, 4, TOK>;
        if (smem > 47 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        mx_launch_chained(kernel, dim3((n_tokens + TOK - 1) / TOK), dim3(vecs > 256 ? 384 : 256), smem, stream, p, cache,
                          q_out, n_tokens);
    } else {
        auto kernel = conv_norm_window_kernel<T, TAPS, 4, 1>;
        if (smem > 47 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        mx_launch_chained(kernel, dim3(n_tokens), dim3(vecs > 256 ? 512 : 256), smem, stream, p, cache, q_out, n_tokens);
    }
    return mx_launch_status();
}

template <typename T>
__global__ void conv_state_update_kernel(const T* __restrict__ rows, int ld, const float* __restrict__ bias,
                                         float* __restrict__ state, long long state_stride,
                                         const int* __restrict__ cu_q, const int* __restrict__ state_slots, int channels,
                                         int taps) {
    const int seq = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    const int first = cu_q[seq], n = cu_q[seq + 1] - first;
    if (c >= channels || n < 2) return;
    float* memory = state + (size_t)state_slots[seq] * state_stride;
    const float b = bias ? bias[c] : 0.f;
    for (int r = 0; r < taps - 1; ++r) {
        // row r becomes the input taps - 1 - r tokens before the next one; rows still to be read lie behind it
        const int local = n - (taps - 1) + r;
        memory[(size_t)r * channels + c] = local >= 0 ? to_float(rows[(size_t)(first + local) * ld + c]) + b
                                                      : memory[(size_t)(n + r) * channels + c];
    }
}

}  // namespace

extern "C" int mx_conv_norm_kv_write(const float* proj, int ld, const float* bias, const float* conv, int taps,
                                     const float* q_weight, const float* k_weight, float eps, float temp_coef,
                                     float temp_every, float* state, long long state_stride, const int* positions,
                                     const int* tok_seq, const int* cu_q, const int* state_slots, const int* slots,
                                     void* cache, long long n_pages, int page_size, void* q_out, int dtype, int n_tokens,
                                     int n_heads, int n_kv_heads, int dim, int vdim, int hd, int own_kv, int* status,
                                     cudaStream_t stream) {
    if (n_tokens <= 0) return MX_OK;
    if (hd < dim || hd < vdim) MX_REFUSE("attention operands: a padded head of %d holds neither %d nor %d", hd, dim, vdim);
    if (taps < 1) MX_REFUSE("convolution: %d taps", taps);
    const int channels = n_heads * dim + (own_kv ? n_kv_heads * (dim + vdim) : 0);
    if (ld < channels) MX_REFUSE("attention operands: projection rows are too short");
    if (state_stride < (long long)(taps - 1) * channels) MX_REFUSE("convolution: a state of %lld floats is too short", state_stride);
    if (!(temp_every > 0.f)) MX_REFUSE("query temperature: a period of %f", temp_every);
    ConvAttnParams p;
    p.proj = proj; p.bias = bias; p.conv = conv; p.q_weight = q_weight; p.k_weight = k_weight; p.state = state;
    p.positions = positions; p.tok_seq = tok_seq; p.cu_q = cu_q; p.state_slots = state_slots;
    p.slots = cache ? slots : nullptr; p.status = status; p.n_slots = n_pages * page_size; p.state_stride = state_stride;
    p.ld = ld; p.taps = taps; p.n_heads = n_heads; p.n_kv_heads = n_kv_heads; p.dim = dim; p.vdim = vdim; p.hd = hd;
    p.page_size = page_size > 0 ? page_size : 1; p.own_kv = own_kv; p.eps = eps; p.temp_coef = temp_coef;
    p.temp_every = temp_every;
    // rows that the 16-byte form takes: widths, strides and addresses in groups of four
    const bool vec = dim % 4 == 0 && vdim % 4 == 0 && ld % 4 == 0 && hd % 4 == 0 && state_stride % 4 == 0 &&
                     ((uintptr_t)proj | (uintptr_t)bias | (uintptr_t)conv | (uintptr_t)state | (uintptr_t)cache |
                      (uintptr_t)q_out) % 16 == 0 && (size_t)channels * sizeof(float) <= 200 * 1024;
#define MX_WINDOW(TAPS)                                                                                              \
    return dtype == MX_DTYPE_F32                                                                                     \
               ? launch_window<float, TAPS>(p, (float*)cache, (float*)q_out, n_tokens, channels, stream)             \
               : launch_window<__nv_bfloat16, TAPS>(p, (__nv_bfloat16*)cache, (__nv_bfloat16*)q_out, n_tokens, channels, \
                                                    stream)
    if (vec && taps == 2) MX_WINDOW(2);
    if (vec && taps == 3) MX_WINDOW(3);
    if (vec && taps == 4) MX_WINDOW(4);
#undef MX_WINDOW
    const size_t smem = (size_t)channels * sizeof(float);
    if (smem > 200 * 1024) MX_REFUSE("attention operands: %d projected channels exceed the 51200 this kernel stages", channels);
    const int threads = 256;
    if (dtype == MX_DTYPE_F32) {
        if (smem > 47 * 1024)
            cudaFuncSetAttribute(conv_norm_kv_write_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        mx_launch_chained(conv_norm_kv_write_kernel<float>, dim3(n_tokens), dim3(threads), smem, stream, p, (float*)cache,
                          (float*)q_out);
    } else {
        if (smem > 47 * 1024)
            cudaFuncSetAttribute(conv_norm_kv_write_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)smem);
        mx_launch_chained(conv_norm_kv_write_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(threads), smem, stream, p,
                          (__nv_bfloat16*)cache, (__nv_bfloat16*)q_out);
    }
    return mx_launch_status();
}

extern "C" int mx_conv_state_update(const void* rows, int dtype, int ld, const float* bias, float* state,
                                    long long state_stride, const int* cu_q, const int* state_slots, int n_seqs,
                                    int channels, int taps, cudaStream_t stream) {
    if (n_seqs <= 0 || channels <= 0 || taps <= 1) return MX_OK;
    const dim3 grid(n_seqs, (channels + 127) / 128);
    if (dtype == MX_DTYPE_F32)
        conv_state_update_kernel<float><<<grid, 128, 0, stream>>>((const float*)rows, ld, bias, state, state_stride, cu_q,
                                                                 state_slots, channels, taps);
    else
        conv_state_update_kernel<__nv_bfloat16><<<grid, 128, 0, stream>>>((const __nv_bfloat16*)rows, ld, bias, state,
                                                                         state_stride, cu_q, state_slots, channels, taps);
    return mx_launch_status();
}
