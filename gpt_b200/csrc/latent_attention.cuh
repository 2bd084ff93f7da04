// Latent attention (multi-head attention whose keys and values are linear maps of one small latent per token).
//
// Only the normed latent c and the rotated key part shared by all heads are cached: a row per position, [c | rotated key] in T, the
// parts padded with zeros.  Two forms of the same attention:
//   absorbed   scores against the cached rows themselves: q_u . (W_uk c) = (W_uk^T q_u) . c, and W_uv is applied to the weighted
//              sum of latents (few rows: decoding, short portions; and all fp32 work)
//   expanded   keys and values of all visible positions as matrices, tensor-core attention over them (prompts)
// Scores, softmax weights and their sums are fp32, rotation angles are formed in fp64.
#pragma once

#include "decoder_rows.cuh"

namespace gptb200 {
namespace dec {

struct LatentShape {
    int heads, dim, rot_dim, vdim, kv_rank;
    int rank_pitch, row_pitch;    // kv_rank padded to 16; cached row [c | rotated key part padded to 16]
    int dim_pad, v_pad;           // rows of W_uk / W_uv per head (dim and vdim padded to 16, zero rows)
    int q_stride;                 // projection columns per head: [unrotated: dim_pad | rotated, padded to 16]
    int rot_half;                 // rotated pairs
    int off_dkv, off_g;           // columns of W_dkv h and W_g h in the projection row (q starts at 0)
    float scale;
    size_t cache_base;            // the cached rows this layer reads (its own or another layer's) start in the slot at
    size_t cache_per_position;    //   cache_base + cache_per_position * capacity
};

template <typename T>
__device__ __forceinline__ T *latent_cache(const LatentShape &s, const StepEntry &e)
{
    return reinterpret_cast<T *>(e.slot + s.cache_base + s.cache_per_position * e.capacity);
}

// cos / sin (times gain) of position * frequency for every row of the step: table[row][pair].
__global__ void rotary_table_kernel(float2 *__restrict__ table, const double *__restrict__ freq, int half, double gain, const StepEntry *__restrict__ entries,
                                    const int *__restrict__ row_entry, int rows)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * half) return;
    const int row = i / half, k = i % half;
    const StepEntry e = entries[row_entry[row]];
    double s, c;
    sincos(static_cast<double>(e.pos0 + row - e.row0) * freq[k], &s, &c);
    table[i] = make_float2(static_cast<float>(c * gain), static_cast<float>(s * gain));
}

// Component k of a rotated part x (rotated pairs, then dimensions that pass unchanged, then zeros for the padding).
template <typename T>
__device__ __forceinline__ float rotated(const T *x, int k, const float2 *cs, const LatentShape &s)
{
    if (k < s.rot_half) return to_f(x[k]) * cs[k].x - to_f(x[k + s.rot_half]) * cs[k].y;
    if (k < 2 * s.rot_half) return to_f(x[k]) * cs[k - s.rot_half].x + to_f(x[k - s.rot_half]) * cs[k - s.rot_half].y;
    return k < s.rot_dim ? to_f(x[k]) : 0.0f;
}

// Per row: rotates the heads' rotated query parts in place; a layer with keys of its own also norms the latent, rotates the shared
// key part and puts both into the cache.
template <typename T>
__global__ void latent_prepare_kernel(T *__restrict__ proj, long long ld, const float2 *__restrict__ table, const float *__restrict__ norm_w, float eps,
                                      const LatentShape s, int own_keys, const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int row0)
{
    __shared__ float red[32];
    grid_dependency_wait();
    grid_dependency_launch();
    const int row = row0 + blockIdx.x;
    const StepEntry e = entries[row_entry[row]];
    T *r = proj + row * ld;
    const float2 *cs = table + static_cast<long long>(row) * s.rot_half;
    for (int i = threadIdx.x; i < s.heads * s.rot_half; i += blockDim.x) {
        const int h = i / s.rot_half, k = i % s.rot_half;
        T *q = r + h * s.q_stride + s.dim_pad + k;
        const float u = to_f(q[0]), v = to_f(q[s.rot_half]);
        q[0] = from_f<T>(u * cs[k].x - v * cs[k].y);
        q[s.rot_half] = from_f<T>(v * cs[k].x + u * cs[k].y);
    }
    if (!own_keys) return;
    const T *d = r + s.off_dkv;
    T *dst = latent_cache<T>(s, e) + static_cast<long long>(e.pos0 + row - e.row0) * s.row_pitch;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < s.kv_rank; i += blockDim.x) {
        const float v = to_f(d[i]);
        ss = fmaf(v, v, ss);
    }
    const float inv = rsqrtf(block_sum(ss, red) / s.kv_rank + eps);
    for (int i = threadIdx.x; i < s.rank_pitch; i += blockDim.x) dst[i] = from_f<T>(i < s.kv_rank ? to_f(d[i]) * inv * norm_w[i] : 0.0f);
    const T *kr = d + s.kv_rank;
    T *kd = dst + s.rank_pitch;
    for (int k = threadIdx.x; k < s.row_pitch - s.rank_pitch; k += blockDim.x) kd[k] = from_f<T>(rotated(kr, k, cs, s));
}

constexpr int kLatentWarps = 4;

// Absorbed form for fp32 work, one block per (head, row): the query is mapped into the latent space, every warp goes through every fourth
// visible position with a running maximum and sum, the warps' parts are merged, W_uv and the output gate are applied.
// NR: cached row values per lane.  w_uk [heads * dim_pad][rank_pitch], w_uv [heads * v_pad][rank_pitch].
template <typename T, int NR>
__global__ void __launch_bounds__(kLatentWarps * 32)
latent_rows_kernel(T *__restrict__ out, int ld_out, const T *__restrict__ proj, long long ld, const T *__restrict__ w_uk, const T *__restrict__ w_uv,
                   const LatentShape s, const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int row0)
{
    extern __shared__ float sm[];
    float *q = sm;                                   // [row_pitch] query in the cached rows' space
    float *acc_sm = q + s.row_pitch;                 // [warps][rank_pitch]
    float *ml = acc_sm + kLatentWarps * s.rank_pitch;   // [warps][2]
    grid_dependency_wait();
    grid_dependency_launch();
    const int h = blockIdx.x, row = row0 + blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const StepEntry e = entries[row_entry[row]];
    const int last = e.pos0 + row - e.row0;          // this row's position
    const T *qr = proj + row * ld + h * s.q_stride;
    for (int j = threadIdx.x; j < s.row_pitch; j += blockDim.x) {
        float v = 0.0f;
        if (j < s.kv_rank) {
            const T *w = w_uk + static_cast<long long>(h) * s.dim_pad * s.rank_pitch + j;
            for (int d = 0; d < s.dim; ++d) v = fmaf(to_f(qr[d]), to_f(w[static_cast<long long>(d) * s.rank_pitch]), v);
        } else if (j >= s.rank_pitch && j - s.rank_pitch < s.rot_dim) {
            v = to_f(qr[s.dim_pad + j - s.rank_pitch]);
        }
        q[j] = v * s.scale;
    }
    __syncthreads();
    float qv[NR], acc[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        qv[i] = lane + 32 * i < s.row_pitch ? q[lane + 32 * i] : 0.0f;
        acc[i] = 0.0f;
    }
    float m = -FLT_MAX, l = 0.0f;
    const T *cache = latent_cache<T>(s, e);
    for (int j = warp; j <= last; j += kLatentWarps) {
        const T *c = cache + static_cast<long long>(j) * s.row_pitch;
        float cv[NR], dot = 0.0f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            cv[i] = lane + 32 * i < s.row_pitch ? to_f(c[lane + 32 * i]) : 0.0f;
            dot = fmaf(qv[i], cv[i], dot);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
        const float mn = fmaxf(m, dot), keep = expf(m - mn), w = expf(dot - mn);
        m = mn;
        l = fmaf(l, keep, w);
#pragma unroll
        for (int i = 0; i < NR; ++i) acc[i] = fmaf(acc[i], keep, w * cv[i]);
    }
#pragma unroll
    for (int i = 0; i < NR; ++i)
        if (lane + 32 * i < s.rank_pitch) acc_sm[warp * s.rank_pitch + lane + 32 * i] = acc[i];
    if (lane == 0) {
        ml[2 * warp] = m;
        ml[2 * warp + 1] = l;
    }
    __syncthreads();
    float top = ml[0];
    for (int w = 1; w < kLatentWarps; ++w) top = fmaxf(top, ml[2 * w]);
    float sum = 0.0f, f[kLatentWarps];
#pragma unroll
    for (int w = 0; w < kLatentWarps; ++w) {
        f[w] = expf(ml[2 * w] - top);
        sum = fmaf(ml[2 * w + 1], f[w], sum);
    }
    for (int j = threadIdx.x; j < s.rank_pitch; j += blockDim.x) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kLatentWarps; ++w) v = fmaf(acc_sm[w * s.rank_pitch + j], f[w], v);
        q[j] = v / sum;   // the query is no longer needed: latent average
    }
    __syncthreads();
    for (int n = warp; n < s.vdim; n += kLatentWarps) {
        const T *w = w_uv + (static_cast<long long>(h) * s.v_pad + n) * s.rank_pitch;
        float v = 0.0f;
        for (int j = lane; j < s.kv_rank; j += 32) v = fmaf(to_f(w[j]), q[j], v);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        if (lane == 0) {
            const float gate = to_f(proj[row * ld + s.off_g + h * s.vdim + n]);
            out[static_cast<long long>(row) * ld_out + h * s.vdim + n] = from_f<T>(v * sigmoid_f(gate));
        }
    }
}

}  // namespace dec
}  // namespace gptb200
