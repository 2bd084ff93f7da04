// Row kernels of the decoder models: embedding, norms around the sublayers, token shift, per-layer token input, depth average,
// sampling.  The residual stream, the norms and everything between them are fp32; T is the type of the activations that enter
// the matrix products (float or bf16).
//
// Row pitch of the stream is the width rounded up to a multiple of 8; the padding columns hold zeros (zero rows and columns of the
// weights, zero norm parameters keep them so).
#pragma once

#include <cfloat>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "gemv_bf16.cuh"

namespace gptb200 {
namespace dec {

// One request's share of a step: `count` rows from row0 on are its tokens at positions pos0, pos0 + 1, ...  Its state lives in
// `slot`.  States that a step reads and replaces from different blocks exist twice; `parity` says which copy is current.
struct StepEntry {
    char *slot;
    int row0, count, pos0, parity;
    int capacity;   // positions the slot's caches can hold
};

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ void store4(float *dst, float4 v) { *reinterpret_cast<float4 *>(dst) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *dst, float4 v)
{
    *reinterpret_cast<uint2 *>(dst) = make_uint2(ptx::pack_bf16x2(v.x, v.y), ptx::pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float4 load4(const float *src) { return *reinterpret_cast<const float4 *>(src); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *src)
{
    const uint2 w = *reinterpret_cast<const uint2 *>(src);
    return make_float4(bf16_lo(w.x), bf16_hi(w.x), bf16_lo(w.y), bf16_hi(w.y));
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// silu where its result is rounded to T: fast exponential and division (2 - 3 ulp of fp32) when that is bf16
template <typename T> __device__ __forceinline__ float silu_t(float z) { return silu_f(z); }
template <> __device__ __forceinline__ float silu_t<__nv_bfloat16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_f(float x) { return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x))); }

// Sum over the block; every thread gets it.  red: 32 floats of shared memory.
__device__ __forceinline__ float block_sum(float v, float *red)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    const int warps = (blockDim.x + 31) >> 5;
    __syncthreads();   // the previous use of `red` is over
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = (threadIdx.x & 31) < warps ? red[threadIdx.x & 31] : 0.0f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    return s;
}

template <typename T>
__global__ void embed_rows_kernel(float *__restrict__ x, const T *__restrict__ table, const int *__restrict__ tokens, int pitch)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const T *src = table + static_cast<long long>(tokens[blockIdx.x]) * pitch;
    float *dst = x + static_cast<long long>(blockIdx.x) * pitch;
    for (int d = 4 * threadIdx.x; d < pitch; d += 4 * blockDim.x) store4(dst + d, load4(src + d));
}

// The same for sequences whose embedding looks one token back: scale * table row + the row of `pairs` that the previous and the
// current token hash to (a sequence's first token: the row after the hashed ones).  The last token of a portion stays in the
// sequence's state (`previous`: offset of int [2]).
template <typename T>
__global__ void embed_pair_rows_kernel(float *__restrict__ x, const T *__restrict__ table, float scale, const T *__restrict__ pairs, long long buckets, long long mul_previous,
                                       long long mul_current, const int *__restrict__ tokens, int pitch, size_t previous, const StepEntry *__restrict__ entries,
                                       const int *__restrict__ row_entry)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const int row = blockIdx.x, token = tokens[row];
    const StepEntry e = entries[row_entry[row]];
    int *state = reinterpret_cast<int *>(e.slot + previous);
    const T *pair = nullptr;
    if (buckets > 0) {
        long long at = buckets;
        if (row > e.row0 || e.pos0 > 0) at = ((row > e.row0 ? tokens[row - 1] : state[e.parity]) * mul_previous + token * mul_current) % buckets;
        pair = pairs + at * pitch;
        if (threadIdx.x == 0 && row == e.row0 + e.count - 1) state[e.parity ^ 1] = token;
    }
    const T *src = table + static_cast<long long>(token) * pitch;
    float *dst = x + static_cast<long long>(row) * pitch;
    for (int d = 4 * threadIdx.x; d < pitch; d += 4 * blockDim.x) {
        float4 v = load4(src + d);
        v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
        if (pair) {
            const float4 b = load4(pair + d);
            v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
        }
        store4(dst + d, v);
    }
}

template <typename T>
struct LayerBegin {
    int rows, width, pitch;
    float eps;
    const float *x_in;        // residual after the previous layer's feed-forward (or the embedding output)
    const float *side_y;      // projected per-layer token input, null: none
    const float *side_w;
    float *states;            // [j][rows][pitch] results of the layers so far (j = 0: embedding output)
    long long state_stride;
    int n_states;             // states that enter the average, the one written here included; 0: no average
    const float *coef;        // [n_states]
    float *x_out;             // residual that enters this layer
    const float *norm_w, *norm_b;
    const float *shift;       // token shift, null: none
    size_t shift_state;       // offset in the slot: [2][pitch] floats, the previous token's normed residual
    T *h;
    const StepEntry *entries;
    const int *row_entry;
    const int *row_list;      // null: all rows; else only these (no shift then), h is packed
    int tile;                 // consecutive rows per block
};

// Start of a layer: the previous layer's token input and result, the depth average, the norm and the token shift in one pass.
// A block takes `tile` consecutive rows; the normed residual of the row before its first one is computed a second time
// (nothing is exchanged between blocks), or comes from the sequence's state.
template <typename T>
__global__ void layer_begin_kernel(const LayerBegin<T> p)
{
    extern __shared__ float sm[];
    float *x = sm, *before = sm + p.pitch;   // this row / previous row's normed values; every thread touches its own columns only
    __shared__ float red[32];
    grid_dependency_wait();
    grid_dependency_launch();

    auto row_normed = [&](int row, bool write, float *dst) {
        const long long at = static_cast<long long>(row) * p.pitch;
        float inv = 0.0f;
        if (p.side_y) {
            float ss = 0.0f;
            for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
                const float4 y = load4(p.side_y + at + d);
                ss += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
            }
            inv = rsqrtf(block_sum(ss, red) / p.width + p.eps);
        }
        float sum = 0.0f;
        for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
            float4 v = load4(p.x_in + at + d);
            if (p.side_y) {
                const float4 y = load4(p.side_y + at + d), w = load4(p.side_w + d);
                v.x += y.x * inv * w.x; v.y += y.y * inv * w.y; v.z += y.z * inv * w.z; v.w += y.w * inv * w.w;
            }
            if (p.n_states > 0) {
                if (write) store4(p.states + (p.n_states - 1) * p.state_stride + at + d, v);
                const float c = p.coef[p.n_states - 1];
                float4 a = make_float4(c * v.x, c * v.y, c * v.z, c * v.w);
                const float *s = p.states + at + d;
#pragma unroll 4
                for (int j = 0; j < p.n_states - 1; ++j, s += p.state_stride) {
                    const float4 u = load4(s);
                    const float cj = p.coef[j];
                    a.x += cj * u.x; a.y += cj * u.y; a.z += cj * u.z; a.w += cj * u.w;
                }
                v = a;
            }
            if (write && p.x_out) store4(p.x_out + at + d, v);
            store4(dst + d, v);
            sum += v.x + v.y + v.z + v.w;
        }
        const float mean = block_sum(sum, red) / p.width;
        float var = 0.0f;
        for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
            const float4 v = load4(dst + d);
            const float e[4] = {v.x - mean, v.y - mean, v.z - mean, v.w - mean};
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (d + k < p.width) var += e[k] * e[k];
        }
        const float rstd = rsqrtf(block_sum(var, red) / p.width + p.eps);
        for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
            const float4 v = load4(dst + d), w = load4(p.norm_w + d), b = load4(p.norm_b + d);
            store4(dst + d, make_float4((v.x - mean) * rstd * w.x + b.x, (v.y - mean) * rstd * w.y + b.y, (v.z - mean) * rstd * w.z + b.z,
                                        (v.w - mean) * rstd * w.w + b.w));
        }
    };

    const int first = blockIdx.x * p.tile;
    if (p.shift) {
        const StepEntry e = p.entries[p.row_entry[first]];
        if (first > e.row0) row_normed(first - 1, false, before);
    }
    for (int i = first; i < min(first + p.tile, p.rows); ++i) {
        const int row = p.row_list ? p.row_list[i] : i;
        row_normed(row, true, x);
        T *h = p.h + static_cast<long long>(i) * p.pitch;
        if (p.shift) {
            const StepEntry e = p.entries[p.row_entry[row]];
            float *state = reinterpret_cast<float *>(e.slot + p.shift_state);
            const float *old = state + e.parity * p.pitch;
            float *next = state + (e.parity ^ 1) * p.pitch;
            const bool from_state = row == e.row0, last = row == e.row0 + e.count - 1;
            for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
                const float4 v = load4(x + d), b = from_state ? load4(old + d) : load4(before + d), m = load4(p.shift + d);
                store4(h + d, make_float4(v.x + (b.x - v.x) * m.x, v.y + (b.y - v.y) * m.y, v.z + (b.z - v.z) * m.z, v.w + (b.w - v.w) * m.w));
                if (last) store4(next + d, v);
            }
            float *t = x;
            x = before;
            before = t;
        } else {
            for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) store4(h + d, load4(x + d));
        }
    }
}

// End of a sublayer: x += layer_norm(y); out = layer_norm(x) for the next sublayer, or x itself (norm2_w null), as T.
template <typename T>
__global__ void sublayer_end_kernel(float *__restrict__ x, const float *__restrict__ y, const float *__restrict__ norm1_w, const float *__restrict__ norm1_b,
                                    const float *__restrict__ norm2_w, const float *__restrict__ norm2_b, T *__restrict__ out, int width, int pitch, float eps)
{
    extern __shared__ float sm[];   // [pitch], every thread its own columns
    __shared__ float red[32];
    grid_dependency_wait();
    grid_dependency_launch();
    const long long at = static_cast<long long>(blockIdx.x) * pitch;
    auto statistics = [&](float sum, float &mean, float &rstd) {
        mean = block_sum(sum, red) / width;
        float var = 0.0f;
        for (int d = 4 * threadIdx.x; d < pitch; d += 4 * blockDim.x) {
            const float4 v = load4(sm + d);
            const float e[4] = {v.x - mean, v.y - mean, v.z - mean, v.w - mean};
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (d + k < width) var += e[k] * e[k];
        }
        rstd = rsqrtf(block_sum(var, red) / width + eps);
    };
    float sum = 0.0f, mean, rstd;
    for (int d = 4 * threadIdx.x; d < pitch; d += 4 * blockDim.x) {
        const float4 v = load4(y + at + d);
        store4(sm + d, v);
        sum += v.x + v.y + v.z + v.w;
    }
    statistics(sum, mean, rstd);
    sum = 0.0f;
    for (int d = 4 * threadIdx.x; d < pitch; d += 4 * blockDim.x) {
        const float4 v = load4(sm + d), w = load4(norm1_w + d), b = load4(norm1_b + d);
        float4 r = load4(x + at + d);
        r.x += (v.x - mean) * rstd * w.x + b.x;
        r.y += (v.y - mean) * rstd * w.y + b.y;
        r.z += (v.z - mean) * rstd * w.z + b.z;
        r.w += (v.w - mean) * rstd * w.w + b.w;
        store4(x + at + d, r);
        store4(sm + d, r);
        sum += r.x + r.y + r.z + r.w;
    }
    if (norm2_w) statistics(sum, mean, rstd);
    for (int d = 4 * threadIdx.x; d < pitch; d += 4 * blockDim.x) {
        float4 v = load4(sm + d);
        if (norm2_w) {
            const float4 w = load4(norm2_w + d), b = load4(norm2_b + d);
            v = make_float4((v.x - mean) * rstd * w.x + b.x, (v.y - mean) * rstd * w.y + b.y, (v.z - mean) * rstd * w.z + b.z, (v.w - mean) * rstd * w.w + b.w);
        }
        store4(out + at + d, v);
    }
}

template <typename T>
struct ResidualNorm {
    int rows, width, pitch;
    float eps, mult;
    const float *x_in;        // residual stream
    const float *y;           // result of the sublayer before, null: none
    float *x_out;             // x_in + mult * y (another buffer than x_in), null: not stored
    const float *norm_w;      // the factor itself
    int mixes;                // 0: h is the normed row; else h holds that many blends of it with the previous token's, mix_stride apart
    const float *mix;         // [mixes][pitch] share of the previous token's
    size_t shift_state;       // offset in the slot: [2][pitch] floats, the previous token's normed row
    long long mix_stride;
    T *h;
    const StepEntry *entries;
    const int *row_entry;
    const int *row_list;      // null: all rows; else only these (no mixes then), h is packed
    int tile;                 // consecutive rows per block
};

// Between sublayers without norms of their own results: x += mult * y, h = x / root mean square * weight, and the blends of h with the
// previous token's where the next mixer reads such.  As in layer_begin_kernel the row before a block's first is computed twice.
template <typename T>
__global__ void residual_norm_kernel(const ResidualNorm<T> p)
{
    extern __shared__ float sm[];
    float *x = sm, *before = sm + p.pitch;   // this row / previous row's normed values; every thread touches its own columns only
    __shared__ float red[32];
    grid_dependency_wait();
    grid_dependency_launch();

    auto row_normed = [&](int row, bool write, float *dst) {
        const long long at = static_cast<long long>(row) * p.pitch;
        float ss = 0.0f;
        for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
            float4 v = load4(p.x_in + at + d);
            if (p.y) {
                const float4 y = load4(p.y + at + d);
                v.x = fmaf(p.mult, y.x, v.x); v.y = fmaf(p.mult, y.y, v.y); v.z = fmaf(p.mult, y.z, v.z); v.w = fmaf(p.mult, y.w, v.w);
            }
            if (write && p.x_out) store4(p.x_out + at + d, v);
            store4(dst + d, v);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        const float inv = rsqrtf(block_sum(ss, red) / p.width + p.eps);
        for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
            const float4 v = load4(dst + d), w = load4(p.norm_w + d);
            store4(dst + d, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
        }
    };

    const int first = blockIdx.x * p.tile;
    if (p.mixes) {
        const StepEntry e = p.entries[p.row_entry[first]];
        if (first > e.row0) row_normed(first - 1, false, before);
    }
    for (int i = first; i < min(first + p.tile, p.rows); ++i) {
        const int row = p.row_list ? p.row_list[i] : i;
        row_normed(row, true, x);
        T *h = p.h + static_cast<long long>(i) * p.pitch;
        if (!p.mixes) {
            for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) store4(h + d, load4(x + d));
            continue;
        }
        const StepEntry e = p.entries[p.row_entry[row]];
        float *state = reinterpret_cast<float *>(e.slot + p.shift_state);
        const float *old = state + e.parity * p.pitch;
        float *next = state + (e.parity ^ 1) * p.pitch;
        const bool from_state = row == e.row0, last = row == e.row0 + e.count - 1;
        for (int d = 4 * threadIdx.x; d < p.pitch; d += 4 * blockDim.x) {
            const float4 v = load4(x + d), b = from_state ? load4(old + d) : load4(before + d);
            for (int k = 0; k < p.mixes; ++k) {
                const float4 m = load4(p.mix + k * p.pitch + d);
                store4(h + k * p.mix_stride + d, make_float4(v.x + (b.x - v.x) * m.x, v.y + (b.y - v.y) * m.y, v.z + (b.z - v.z) * m.z, v.w + (b.w - v.w) * m.w));
            }
            if (last) store4(next + d, v);
        }
        float *t = x;
        x = before;
        before = t;
    }
}

// A row of a mixer's output divided by its root mean square, times weight, times sigmoid(gate), as T.
template <typename T>
__global__ void normed_sigmoid_gate_kernel(T *__restrict__ out, int ld_out, const float *__restrict__ y, int width, const T *__restrict__ gate, long long ld_gate,
                                           const float *__restrict__ weight, float eps)
{
    extern __shared__ float sm[];   // [width], every thread its own columns
    __shared__ float red[32];
    grid_dependency_wait();
    grid_dependency_launch();
    const long long row = blockIdx.x;
    y += row * width;
    gate += row * ld_gate;
    out += row * ld_out;
    float ss = 0.0f;
    if (width % 4 == 0) {
        for (int i = 4 * threadIdx.x; i < width; i += 4 * blockDim.x) {
            const float4 v = load4(y + i);
            store4(sm + i, v);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        const float inv = rsqrtf(block_sum(ss, red) / width + eps);
        for (int i = 4 * threadIdx.x; i < width; i += 4 * blockDim.x) {
            const float4 v = load4(sm + i), w = load4(weight + i), g = load4(gate + i);
            store4(out + i, make_float4(v.x * inv * w.x * sigmoid_f(g.x), v.y * inv * w.y * sigmoid_f(g.y), v.z * inv * w.z * sigmoid_f(g.z), v.w * inv * w.w * sigmoid_f(g.w)));
        }
        return;
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        sm[i] = y[i];
        ss = fmaf(sm[i], sm[i], ss);
    }
    const float inv = rsqrtf(block_sum(ss, red) / width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) out[i] = from_f<T>(sm[i] * inv * weight[i] * sigmoid_f(to_f(gate[i])));
}

// Unfused tails of the fp32 products (the bf16 products do these in their epilogues).
// act[row][j] = gelu(gate) * up, or silu(gate) * up, from columns in groups of 32 gate | 32 up
__global__ void glu_rows_kernel(float *__restrict__ act, const float *__restrict__ in, int columns, long long ld_in, bool silu)
{
    const float *src = in + blockIdx.x * ld_in;
    float *dst = act + static_cast<long long>(blockIdx.x) * columns;
    for (int j = threadIdx.x; j < columns; j += blockDim.x) {
        const int g = (j >> 5) * 64 + (j & 31);
        dst[j] = (silu ? silu_f(src[g]) : gelu_f(src[g])) * src[g + 32];
    }
}

__global__ void silu_columns_kernel(float *__restrict__ x, int columns, long long ld)
{
    float *r = x + blockIdx.x * ld;
    for (int j = threadIdx.x; j < columns; j += blockDim.x) r[j] = silu_f(r[j]);
}

__global__ void gelu_factor_rows_kernel(float *__restrict__ x, const float *__restrict__ factor, const int *__restrict__ factor_rows, int columns)
{
    float *r = x + static_cast<long long>(blockIdx.x) * columns;
    const float *f = factor + static_cast<long long>(factor_rows[blockIdx.x]) * columns;
    for (int j = threadIdx.x; j < columns; j += blockDim.x) r[j] = gelu_f(r[j]) * f[j];
}

// ---- sampling ------------------------------------------------------------------------------------------------------
// 32 well-mixed bits of a counter (splitmix64 finaliser).
__device__ __forceinline__ unsigned int mix_bits(unsigned long long z)
{
    z += 0x9E3779B97F4A7C15ull;
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    return static_cast<unsigned int>((z ^ (z >> 31)) >> 32);
}

// What a generation step reads and advances in device memory.
struct GenerateControl {
    unsigned long long seed;
    int step;
    float temperature;
};

// One token per row of logits: the largest logit (temperature 0; the first of equals), or a draw from softmax(logits / temperature)
// by the Gumbel-max rule: argmax of logit / temperature - log(-log(u)).
__device__ __forceinline__ int sample_row(const float *__restrict__ row, int vocab, float temperature, unsigned long long seed, unsigned long long draw)
{
    __shared__ float best_v[32];
    __shared__ int best_i[32];
    float bv = -FLT_MAX;
    int bi = 0x7fffffff;
    for (int i = threadIdx.x; i < vocab; i += blockDim.x) {
        float v = row[i];
        if (temperature > 0.0f) {
            const unsigned long long counter = draw * 0x100000000ull + i;
            const float u = (mix_bits(seed ^ mix_bits(counter) ^ (counter << 20)) + 0.5f) * 2.3283064365386963e-10f;
            v = v / temperature - logf(-logf(fminf(u, 0.99999994f)));
        }
        if (v > bv || (v == bv && i < bi)) {
            bv = v;
            bi = i;
        }
    }
    auto merge = [&](float v, int i) {
        if (v > bv || (v == bv && i < bi)) {
            bv = v;
            bi = i;
        }
    };
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, bv, o);
        const int i = __shfl_xor_sync(0xffffffffu, bi, o);
        merge(v, i);
    }
    if ((threadIdx.x & 31) == 0) {
        best_v[threadIdx.x >> 5] = bv;
        best_i[threadIdx.x >> 5] = bi;
    }
    __syncthreads();
    if (threadIdx.x == 0)
        for (int w = 1; w < static_cast<int>(blockDim.x >> 5); ++w) merge(best_v[w], best_i[w]);
    return min(bi, vocab - 1);   // thread 0's is the block's
}

__global__ void sample_rows_kernel(int *__restrict__ tokens, const float *__restrict__ logits, int vocab, long long pitch, float temperature,
                                   unsigned long long seed, unsigned long long draw)
{
    const int t = sample_row(logits + blockIdx.x * pitch, vocab, temperature, seed, draw * gridDim.x + blockIdx.x);
    if (threadIdx.x == 0) tokens[blockIdx.x] = t;
}

// The same inside a generation step: the token goes to the next step's input and to history [step][sequence], and the sequence's
// entry moves on by one position.
__global__ void sample_advance_kernel(int *__restrict__ tokens, int *__restrict__ history, const GenerateControl *__restrict__ control, const float *__restrict__ logits,
                                      int vocab, long long pitch, StepEntry *__restrict__ entries)
{
    grid_dependency_wait();
    const GenerateControl c = *control;
    const int t = sample_row(logits + blockIdx.x * pitch, vocab, c.temperature, c.seed, static_cast<unsigned long long>(c.step) * gridDim.x + blockIdx.x);
    if (threadIdx.x == 0) {
        tokens[blockIdx.x] = t;
        history[static_cast<long long>(c.step) * gridDim.x + blockIdx.x] = t;
        entries[blockIdx.x].pos0 += 1;
        entries[blockIdx.x].parity ^= 1;
    }
}

__global__ void advance_step_kernel(GenerateControl *control)
{
    grid_dependency_wait();
    control->step += 1;
}

}  // namespace dec
}  // namespace gptb200
