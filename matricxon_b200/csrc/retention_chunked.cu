// Retention over long portions, chunk by chunk: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T (q_scale q_t), every head's o
// divided by its root mean square and multiplied by silu(gate), q and k rotated over their first entries.
//
// The decay is one constant per head, so a chunk of 64 tokens is three small products on the FP32 cores (float operands and
// sums: the recurrence stays in 32-bit) instead of 64 rank-one updates:
//   retention_maps     per (chunk, head): what the chunk adds to the state by its end, sum_j decay^(n-1-j) k_j v_j^T
//   retention_carry    per (sequence, head): the chunks' start states in order, from and to the state slot
//   retention_outputs  per (chunk, head): o_i = q_scale (decay^(i+1) q_i S_start + sum_(j<=i) decay^(i-j) (q_i . k_j) v_j),
//                      then the norm, the gate and the rounding, so that o never reaches memory
// A block holds the chunk's q, k and v rows in shared memory (rotated in place: pairs (i, i + rot/2), angle
// position * freq[i] in float), and its start state in the keys' place once the scores exist (two blocks an SM); 256 threads own 4 x 8 pieces of the outputs (8 x 8 of a map). Heads of up to 128 key
// channels and 128 values, padded with zeros to 64 or 128. Rows of tokens that the chunk does not have are skipped.
// `silu`: q, k and v are the silu of what the projection holds. `raw`: o itself goes out, in float, without norm and gate.
// Equal to the token-by-token recurrence up to float rounding, however the sequence was cut.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int RC_TOKENS = 64, RC_THREADS = 256, RC_PAD = 4;

struct RetentionParams {
    const float* proj;          // rows [.. q | k | v | gate ..], `ld` floats apart
    const float* decay;         // [heads]
    const int* positions;
    const float* freq;          // null: no rotation
    const int* cu_q;
    const int* state_slots;
    const int* chunks;          // [n_chunks][2]: (sequence, first token within its portion)
    const int* seq_chunk0;      // [n_seqs + 1]
    float* state;               // [slots][heads][dim][vdim]
    float* chunk_state;         // [n_chunks][heads][dim][vdim]: what a chunk adds, then its start state
    int ld, q_col, k_col, v_col, g_col, heads, dim, vdim, rot, out_ld;
    float q_scale, eps;
    int silu, raw;
    int vec;                    // widths, strides and columns in groups of four
};

// rows of one head ([tokens][width] at column `col`) into shared memory [RC_TOKENS][P + RC_PAD], zeros beyond `n` and `width`
template <int P>
__device__ __forceinline__ void load_rows(float* dst, const float* src, int ld, int n, int width, int vec, int silu = 0) {
    constexpr int S = P + RC_PAD;
    if (vec) {
        constexpr int ITEMS = RC_TOKENS * (P / 4) / RC_THREADS;
        float4 v[ITEMS];                                     // all of a thread's loads set out before the first is stored
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int item = threadIdx.x + i * RC_THREADS, j = item / (P / 4), c = (item % (P / 4)) * 4;
            v[i] = j < n && c < width ? *reinterpret_cast<const float4*>(src + (size_t)j * ld + c)
                                      : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int item = threadIdx.x + i * RC_THREADS, j = item / (P / 4), c = (item % (P / 4)) * 4;
            if (silu) v[i] = make_float4(silu_of<float>(v[i].x), silu_of<float>(v[i].y), silu_of<float>(v[i].z), silu_of<float>(v[i].w));
            *reinterpret_cast<float4*>(dst + j * S + c) = v[i];
        }
    } else {
        for (int item = threadIdx.x; item < RC_TOKENS * P; item += RC_THREADS) {
            const int j = item / P, c = item % P;
            const float v = j < n && c < width ? src[(size_t)j * ld + c] : 0.f;
            dst[j * S + c] = silu ? silu_of<float>(v) : v;
        }
    }
}

// rotates rows of `a` (and of `b`, if there is one) in place
template <int P>
__device__ __forceinline__ void rotate_rows(float* a, float* b, const int* positions, const float* freq, int rot, int n) {
    constexpr int S = P + RC_PAD;
    const int half = rot >> 1;
    for (int item = threadIdx.x; item < n * half; item += RC_THREADS) {
        const int j = item / half, i = item - j * half;
        float sn, cs;
        sincosf((float)positions[j] * freq[i], &sn, &cs);
        float* p = a + j * S + i;
        const float u = p[0], v = p[half];
        p[0] = u * cs - v * sn;
        p[half] = v * cs + u * sn;
        if (b) {
            float* r = b + j * S + i;
            const float x = r[0], y = r[half];
            r[0] = x * cs - y * sn;
            r[half] = y * cs + x * sn;
        }
    }
}

__device__ __forceinline__ void fma4(float4& acc, float a, const float4& b) {
    acc.x = fmaf(a, b.x, acc.x); acc.y = fmaf(a, b.y, acc.y); acc.z = fmaf(a, b.z, acc.z); acc.w = fmaf(a, b.w, acc.w);
}

template <int DP, int VP>
__global__ void __launch_bounds__(RC_THREADS)
retention_maps_kernel(const RetentionParams p) {
    extern __shared__ __align__(16) float rc_smem[];
    constexpr int KS = DP + RC_PAD, VS = VP + RC_PAD;
    float* k_s = rc_smem;                                    // [RC_TOKENS][KS]
    float* v_s = k_s + RC_TOKENS * KS;                       // [RC_TOKENS][VS]
    __shared__ float power[RC_TOKENS];
    const int chunk = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
    const int seq = p.chunks[2 * chunk], t0 = p.cu_q[seq] + p.chunks[2 * chunk + 1];
    const int n = min(RC_TOKENS, p.cu_q[seq + 1] - t0);
    const float* rows = p.proj + (size_t)t0 * p.ld;
    load_rows<DP>(k_s, rows + p.k_col + head * p.dim, p.ld, n, p.dim, p.vec, p.silu);
    load_rows<VP>(v_s, rows + p.v_col + head * p.vdim, p.ld, n, p.vdim, p.vec, p.silu);
    if (tid < RC_TOKENS) power[tid] = powf(p.decay[head], (float)max(n - 1 - tid, 0));
    __syncthreads();
    if (p.freq) {
        rotate_rows<DP>(k_s, nullptr, p.positions + t0, p.freq, p.rot, n);
        __syncthreads();
    }
    for (int item = tid; item < RC_TOKENS * (VP / 4); item += RC_THREADS) {
        const int j = item / (VP / 4);
        float4* v = reinterpret_cast<float4*>(v_s + j * VS + (item % (VP / 4)) * 4);
        const float w = power[j];
        *v = make_float4(v->x * w, v->y * w, v->z * w, v->w * w);
    }
    __syncthreads();
    // a thread owns DP/16 x VP/16 of the map: rows RA ty .. RA ty + RA - 1, columns 4 tx + 64 b .. + 3
    constexpr int RA = DP / 16, CB = VP / 64;
    const int ty = tid >> 4, tx = tid & 15;
    float4 acc[RA][CB];
#pragma unroll
    for (int a = 0; a < RA; ++a)
#pragma unroll
        for (int b = 0; b < CB; ++b) acc[a][b] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int j = 0; j < n; ++j) {
        float4 v[CB];
        float k[RA];
#pragma unroll
        for (int b = 0; b < CB; ++b) v[b] = *reinterpret_cast<const float4*>(v_s + j * VS + 4 * tx + 64 * b);
#pragma unroll
        for (int a = 0; a < RA; a += 4)
            *reinterpret_cast<float4*>(k + a) = *reinterpret_cast<const float4*>(k_s + j * KS + RA * ty + a);
#pragma unroll
        for (int a = 0; a < RA; ++a)
#pragma unroll
            for (int b = 0; b < CB; ++b) fma4(acc[a][b], k[a], v[b]);
    }
    float* out = p.chunk_state + ((size_t)chunk * p.heads + head) * p.dim * p.vdim;
#pragma unroll
    for (int a = 0; a < RA; ++a) {
        const int d = RA * ty + a;
        if (d >= p.dim) continue;
#pragma unroll
        for (int b = 0; b < CB; ++b) {
            const int e = 4 * tx + 64 * b;
            const float o[4] = {acc[a][b].x, acc[a][b].y, acc[a][b].z, acc[a][b].w};
            if (p.vec) {
                if (e < p.vdim) *reinterpret_cast<float4*>(out + (size_t)d * p.vdim + e) = acc[a][b];
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (e + x < p.vdim) out[(size_t)d * p.vdim + e + x] = o[x];
            }
        }
    }
}

__global__ void __launch_bounds__(256)
retention_carry_kernel(const RetentionParams p) {
    const int seq = blockIdx.x, head = blockIdx.y;
    const int i = blockIdx.z * blockDim.x + threadIdx.x, count = p.dim * p.vdim;
    const int tokens = p.cu_q[seq + 1] - p.cu_q[seq];
    if (i >= count || tokens <= 0) return;
    const float decay = p.decay[head];
    const float whole = powf(decay, (float)RC_TOKENS);
    float* slot = p.state + ((size_t)p.state_slots[seq] * p.heads + head) * count + i;
    float s = *slot;
    const int first = p.seq_chunk0[seq], end = p.seq_chunk0[seq + 1];
    float* here = p.chunk_state + ((size_t)first * p.heads + head) * count + i;
    const size_t stride = (size_t)p.heads * count;
    constexpr int AHEAD = 8;                                 // what chunks add sets out ahead of the chain that needs it
    float added[AHEAD];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) added[a] = first + a < end ? here[a * stride] : 0.f;
    for (int chunk = first; chunk < end; chunk += AHEAD) {
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            if (chunk + a >= end) break;
            const float mine = added[a];
            if (chunk + a + AHEAD < end) added[a] = here[(a + AHEAD) * stride];
            here[a * stride] = s;
            const int left = tokens - (chunk + a - first) * RC_TOKENS;
            s = fmaf(left >= RC_TOKENS ? whole : powf(decay, (float)left), s, mine);
        }
        here += AHEAD * stride;
    }
    *slot = s;
}

template <typename T, int DP, int VP>
__global__ void __launch_bounds__(RC_THREADS, 2)
retention_outputs_kernel(const RetentionParams p, T* __restrict__ out) {
    extern __shared__ __align__(16) float rc_smem[];
    constexpr int KS = DP + RC_PAD, VS = VP + RC_PAD, PS = RC_TOKENS + RC_PAD;
    float* q_s = rc_smem;                                    // [RC_TOKENS][KS]
    constexpr int MID = RC_TOKENS * (KS > VS ? KS : VS);
    float* k_s = q_s + RC_TOKENS * (KS > PS ? KS : PS);      // keys [RC_TOKENS][KS], then 64 rows of the start state [64][VS]
    float* v_s = k_s + MID;                                  // [RC_TOKENS][VS]
    float* s_s = k_s;
    __shared__ float power[RC_TOKENS + 1];
    const int chunk = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
    const int seq = p.chunks[2 * chunk], t0 = p.cu_q[seq] + p.chunks[2 * chunk + 1];
    const int n = min(RC_TOKENS, p.cu_q[seq + 1] - t0);
    const float* rows = p.proj + (size_t)t0 * p.ld;
    load_rows<DP>(q_s, rows + p.q_col + head * p.dim, p.ld, n, p.dim, p.vec, p.silu);
    load_rows<DP>(k_s, rows + p.k_col + head * p.dim, p.ld, n, p.dim, p.vec, p.silu);
    load_rows<VP>(v_s, rows + p.v_col + head * p.vdim, p.ld, n, p.vdim, p.vec, p.silu);
    const float* start = p.chunk_state + ((size_t)chunk * p.heads + head) * p.dim * p.vdim;
    if (tid <= RC_TOKENS) power[tid] = powf(p.decay[head], (float)tid);
    __syncthreads();
    if (p.freq) {
        rotate_rows<DP>(q_s, k_s, p.positions + t0, p.freq, p.rot, n);
        __syncthreads();
    }
    // a thread owns tokens 4 ty .. 4 ty + 3: scores against keys tx + 16 c, outputs 4 tx + 64 b .. + 3
    const int ty = tid >> 4, tx = tid & 15, row0 = 4 * ty;
    const bool live = row0 < n;
    float score[4][4];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) score[r][c] = 0.f;
    if (live) {
#pragma unroll 2
        for (int d = 0; d < DP; d += 4) {
            float4 q[4];
#pragma unroll
            for (int r = 0; r < 4; ++r) q[r] = *reinterpret_cast<const float4*>(q_s + (row0 + r) * KS + d);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float4 k = *reinterpret_cast<const float4*>(k_s + (tx + 16 * c) * KS + d);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    score[r][c] = fmaf(q[r].x, k.x, score[r][c]); score[r][c] = fmaf(q[r].y, k.y, score[r][c]);
                    score[r][c] = fmaf(q[r].z, k.z, score[r][c]); score[r][c] = fmaf(q[r].w, k.w, score[r][c]);
                }
            }
        }
    }
    constexpr int CB = VP / 64;
    float4 acc[4][CB];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int b = 0; b < CB; ++b) acc[r][b] = make_float4(0.f, 0.f, 0.f, 0.f);
    // q S_start, times decay^(i + 1): the start state takes the keys' place, 64 rows at a time
    for (int d0 = 0; d0 < DP; d0 += 64) {
        __syncthreads();
        load_rows<VP>(s_s, start + (size_t)d0 * p.vdim, p.vdim, max(0, min(64, p.dim - d0)), p.vdim, p.vec);
        __syncthreads();
        if (!live) continue;
#pragma unroll 2
        for (int d = 0; d < 64; d += 4) {
            float q[4][4];
#pragma unroll
            for (int r = 0; r < 4; ++r)
                *reinterpret_cast<float4*>(q[r]) = *reinterpret_cast<const float4*>(q_s + (row0 + r) * KS + d0 + d);
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int b = 0; b < CB; ++b) {
                    const float4 s = *reinterpret_cast<const float4*>(s_s + (d + x) * VS + 4 * tx + 64 * b);
#pragma unroll
                    for (int r = 0; r < 4; ++r) fma4(acc[r][b], q[r][x], s);
                }
        }
    }
    __syncthreads();                                         // the queries are done with: the scores take their place
    float* p_s = q_s;
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int i = row0 + r, j = tx + 16 * c;
            p_s[i * PS + j] = j <= i ? score[r][c] * power[j <= i ? i - j : 0] : 0.f;
        }
    __syncthreads();
    if (!live) return;
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const float w = power[row0 + r + 1];
#pragma unroll
        for (int b = 0; b < CB; ++b) { acc[r][b].x *= w; acc[r][b].y *= w; acc[r][b].z *= w; acc[r][b].w *= w; }
    }
    // the chunk's own tokens up to each row
#pragma unroll 2
    for (int j = 0; j <= row0 + 3; j += 4) {
        float s[4][4];
#pragma unroll
        for (int r = 0; r < 4; ++r) *reinterpret_cast<float4*>(s[r]) = *reinterpret_cast<const float4*>(p_s + (row0 + r) * PS + j);
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int b = 0; b < CB; ++b) {
                const float4 v = *reinterpret_cast<const float4*>(v_s + (j + x) * VS + 4 * tx + 64 * b);
#pragma unroll
                for (int r = 0; r < 4; ++r) fma4(acc[r][b], s[r][x], v);
            }
    }
    // every row's norm over the head's values (16 neighbouring lanes hold a row), the gate, one rounding
    const unsigned row_lanes = 0xffffu << (tid & 16);
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        float squares = 0.f;
#pragma unroll
        for (int b = 0; b < CB; ++b) {
            acc[r][b].x *= p.q_scale; acc[r][b].y *= p.q_scale; acc[r][b].z *= p.q_scale; acc[r][b].w *= p.q_scale;
            squares = fmaf(acc[r][b].x, acc[r][b].x, squares); squares = fmaf(acc[r][b].y, acc[r][b].y, squares);
            squares = fmaf(acc[r][b].z, acc[r][b].z, squares); squares = fmaf(acc[r][b].w, acc[r][b].w, squares);
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) squares += __shfl_xor_sync(row_lanes, squares, o);
        const int i = row0 + r;
        if (i >= n) continue;
        if (p.raw) {
            T* dst = out + (size_t)(t0 + i) * p.out_ld + (size_t)head * p.vdim;
#pragma unroll
            for (int b = 0; b < CB; ++b) {
                const int e = 4 * tx + 64 * b;
                const float o[4] = {acc[r][b].x, acc[r][b].y, acc[r][b].z, acc[r][b].w};
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (e + x < p.vdim) dst[e + x] = from_float<T>(o[x]);
            }
            continue;
        }
        const float inv = 1.0f / sqrtf(squares / (float)p.vdim + p.eps);
        const float* gate = rows + (size_t)i * p.ld + p.g_col + head * p.vdim;
        T* dst = out + (size_t)(t0 + i) * p.out_ld + (size_t)head * p.vdim;
#pragma unroll
        for (int b = 0; b < CB; ++b) {
            const int e = 4 * tx + 64 * b;
            const float o[4] = {acc[r][b].x, acc[r][b].y, acc[r][b].z, acc[r][b].w};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                if (e + x < p.vdim) {
                    const float g = gate[e + x];
                    dst[e + x] = from_float<T>(o[x] * inv * silu_of<T>(g));
                }
            }
        }
    }
}

template <typename T, int DP, int VP>
int launch_retention(const RetentionParams& p, T* out, int n_seqs, int n_chunks, cudaStream_t stream) {
    const size_t maps = (size_t)RC_TOKENS * (DP + RC_PAD + VP + RC_PAD) * sizeof(float);
    constexpr int wide = (DP > VP ? DP : VP) + RC_PAD;
    const size_t outputs = (size_t)RC_TOKENS * (DP + RC_PAD + wide + VP + RC_PAD) * sizeof(float);
    static bool ready = false;
    if (!ready) {
        cudaError_t e = cudaFuncSetAttribute(retention_maps_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)maps);
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(retention_outputs_kernel<T, DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)outputs);
        if (e != cudaSuccess) MX_REFUSE("retention: cannot reserve %zu bytes of shared memory", outputs);
        ready = true;
    }
    retention_maps_kernel<DP, VP><<<dim3(n_chunks, p.heads), RC_THREADS, maps, stream>>>(p);
    retention_carry_kernel<<<dim3(n_seqs, p.heads, (p.dim * p.vdim + 255) / 256), 256, 0, stream>>>(p);
    retention_outputs_kernel<T, DP, VP><<<dim3(n_chunks, p.heads), RC_THREADS, outputs, stream>>>(p, out);
    return mx_launch_status();
}

template <typename T>
int pick_retention(const RetentionParams& p, T* out, int n_seqs, int n_chunks, cudaStream_t stream) {
    if (p.dim <= 64 && p.vdim <= 64) return launch_retention<T, 64, 64>(p, out, n_seqs, n_chunks, stream);
    if (p.dim <= 64) return launch_retention<T, 64, 128>(p, out, n_seqs, n_chunks, stream);
    if (p.vdim <= 64) return launch_retention<T, 128, 64>(p, out, n_seqs, n_chunks, stream);
    return launch_retention<T, 128, 128>(p, out, n_seqs, n_chunks, stream);
}

}  // namespace

extern "C" int mx_retention_chunk_tokens() { return RC_TOKENS; }

// chunks: [n_chunks][2] (sequence, first token within its portion) in chunks of mx_retention_chunk_tokens() tokens, sequence
// by sequence; seq_chunk0: [n_seqs + 1]; scratch: n_chunks * heads * dim * vdim floats.
extern "C" int mx_retention_chunked(const float* proj, int ld, int q_col, int k_col, int v_col, int g_col, const float* decay,
                                    float q_scale, float eps, const int* positions, const float* freq, int rot, float* state,
                                    const int* cu_q, const int* state_slots, int n_seqs, const int* chunks,
                                    const int* seq_chunk0, int n_chunks, float* scratch, void* out, int dtype, int out_ld,
                                    int heads, int dim, int vdim, int silu, int raw, cudaStream_t stream) {
    if (n_seqs <= 0 || n_chunks <= 0) return MX_OK;
    if (dim <= 0 || dim > 128 || vdim <= 0 || vdim > 128) MX_REFUSE("chunked retention: heads of %d x %d (at most 128 x 128)", dim, vdim);
    if (heads <= 0 || heads > 65535) MX_REFUSE("chunked retention: %d heads exceed the grid", heads);
    if (rot < 0 || rot % 2 != 0 || rot > dim) MX_REFUSE("chunked retention: %d rotated entries in a head of %d", rot, dim);
    RetentionParams p;
    p.proj = proj; p.decay = decay; p.positions = positions; p.freq = rot > 0 ? freq : nullptr; p.cu_q = cu_q;
    p.state_slots = state_slots; p.chunks = chunks; p.seq_chunk0 = seq_chunk0; p.state = state; p.chunk_state = scratch;
    p.ld = ld; p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.g_col = g_col; p.heads = heads; p.dim = dim; p.vdim = vdim;
    p.silu = silu; p.raw = raw; p.rot = rot; p.out_ld = out_ld; p.q_scale = q_scale; p.eps = eps;
    p.vec = (dim | vdim | ld | q_col | k_col | v_col) % 4 == 0 && ((uintptr_t)proj | (uintptr_t)scratch) % 16 == 0;
    if (dtype == MX_DTYPE_F32) return pick_retention<float>(p, (float*)out, n_seqs, n_chunks, stream);
    return pick_retention<__nv_bfloat16>(p, (__nv_bfloat16*)out, n_seqs, n_chunks, stream);
}
