// Grouped attention: H query heads over G heads of keys and values (query head h reads key / value head h / (H / G)), neighbouring
// dimensions rotated by position, scores optionally capped, values optionally blended with those of an earlier layer, a sigmoid
// gate on the output.
//
// A layer's projection row is [q: H x dim_pad | k: G x dim_pad | v: G x v_pad | gate: H x vdim] in T, padding columns zero; a cached row
// [k: G x dim_pad | v: G x v_pad] holds rotated keys and blended values.  Three forms:
//   grouped_rows_kernel        fp32: one block per (head, row)
//   grouped_split_kernel       bf16, a few rows (decoding, short portions): ranges of positions side by side, then grouped_combine_kernel
//   attention_prefill_kernel   bf16, prompts: over the cache itself (attention_prefill_sm100.cuh)
// Scores, softmax weights and their sums are fp32, rotation angles are formed in fp64.
#pragma once

#include "latent_attention.cuh"
#include "mamba2_chunk.cuh"   // mma16

namespace gptb200 {
namespace dec {

struct GroupedShape {
    int heads, kv_heads, dim, vdim;
    int dim_pad, v_pad;           // multiples of 16
    int row_pitch;                // cached row
    int off_k, off_v, off_g;      // columns in the projection row (q starts at 0)
    int rot_half;                 // rotated pairs
    float scale, softcap;         // softcap 0: none
    size_t cache_base, cache_per_position;   // as in LatentShape
};

template <typename T>
__device__ __forceinline__ T *grouped_cache(const GroupedShape &s, const StepEntry &e)
{
    return reinterpret_cast<T *>(e.slot + s.cache_base + s.cache_per_position * e.capacity);
}

__device__ __forceinline__ float capped_score(float x, const GroupedShape &s) { return s.softcap > 0.0f ? s.softcap * tanhf(x / s.softcap) : x; }

template <typename T> __device__ __forceinline__ float2 load2(const T *src);
template <> __device__ __forceinline__ float2 load2<float>(const float *src) { return *reinterpret_cast<const float2 *>(src); }
template <> __device__ __forceinline__ float2 load2<__nv_bfloat16>(const __nv_bfloat16 *src)
{
    const uint32_t w = *reinterpret_cast<const uint32_t *>(src);
    return make_float2(bf16_lo(w), bf16_hi(w));
}
__device__ __forceinline__ void store2(float *dst, float a, float b) { *reinterpret_cast<float2 *>(dst) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16 *dst, float a, float b) { *reinterpret_cast<uint32_t *>(dst) = ptx::pack_bf16x2(a, b); }

// Per row: rotates the queries in place, puts rotated keys and values into the cache.  first: [rows][kv_heads * v_pad] values of the first
// layer that blends them; share < 0: this is that layer and leaves them there, else v <- (1 - share) v + share * first (null: no
// blending).
template <typename T>
__global__ void grouped_prepare_kernel(T *__restrict__ proj, long long ld, const float2 *__restrict__ table, T *__restrict__ first, float share, const GroupedShape s,
                                       const StepEntry *__restrict__ entries, const int *__restrict__ row_entry)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const long long row = blockIdx.x;
    const StepEntry e = entries[row_entry[row]];
    T *r = proj + row * ld;
    const float2 *cs = table + row * s.rot_half;
    T *dst = grouped_cache<T>(s, e) + (e.pos0 + row - e.row0) * s.row_pitch;
    for (int i = threadIdx.x; i < s.heads * s.rot_half; i += blockDim.x) {
        const int k = i % s.rot_half;
        T *q = r + i / s.rot_half * s.dim_pad + 2 * k;
        const float2 v = load2(q), c = cs[k];
        store2(q, v.x * c.x - v.y * c.y, v.y * c.x + v.x * c.y);
    }
    const int half = s.dim_pad / 2;
    for (int i = threadIdx.x; i < s.kv_heads * half; i += blockDim.x) {
        const int k = i % half;
        float2 v = load2(r + s.off_k + 2 * i);
        if (k < s.rot_half) {
            const float2 c = cs[k];
            v = make_float2(v.x * c.x - v.y * c.y, v.y * c.x + v.x * c.y);
        }
        store2(dst + 2 * i, v.x, v.y);
    }
    const int values = s.kv_heads * s.v_pad;
    T *keep = first ? first + row * values : nullptr, *vd = dst + s.kv_heads * s.dim_pad;
    for (int i = 2 * threadIdx.x; i < values; i += 2 * blockDim.x) {
        float2 v = load2(r + s.off_v + i);
        if (keep && share < 0.0f) {
            store2(keep + i, v.x, v.y);
        } else if (keep) {
            const float2 f = load2(keep + i);
            v = make_float2((1.0f - share) * v.x + share * f.x, (1.0f - share) * v.y + share * f.y);
        }
        store2(vd + i, v.x, v.y);
    }
}

constexpr int kGroupedWarps = 4;

// fp32 work: every warp goes through every fourth visible position with a running maximum and sum, the warps' parts are merged.
// NR: dimensions (and values) per lane.  grid: (heads, rows)
template <typename T, int NR>
__global__ void __launch_bounds__(kGroupedWarps * 32)
grouped_rows_kernel(T *__restrict__ out, int ld_out, const T *__restrict__ proj, long long ld, const GroupedShape s, const StepEntry *__restrict__ entries, const int *__restrict__ row_entry)
{
    extern __shared__ float sm[];                    // [warps][v_pad]
    __shared__ float ml[kGroupedWarps][2];
    grid_dependency_wait();
    grid_dependency_launch();
    const int h = blockIdx.x;
    const long long row = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const StepEntry e = entries[row_entry[row]];
    const int last = e.pos0 + static_cast<int>(row) - e.row0, g = h / (s.heads / s.kv_heads);
    const T *q = proj + row * ld + h * s.dim_pad;
    const T *keys = grouped_cache<T>(s, e) + g * s.dim_pad, *values = grouped_cache<T>(s, e) + s.kv_heads * s.dim_pad + g * s.v_pad;
    float qv[NR], acc[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        qv[i] = lane + 32 * i < s.dim ? to_f(q[lane + 32 * i]) : 0.0f;
        acc[i] = 0.0f;
    }
    float m = -FLT_MAX, l = 0.0f;
    for (int j = warp; j <= last; j += kGroupedWarps) {
        const T *k = keys + static_cast<long long>(j) * s.row_pitch, *v = values + static_cast<long long>(j) * s.row_pitch;
        float dot = 0.0f;
#pragma unroll
        for (int i = 0; i < NR; ++i)
            if (lane + 32 * i < s.dim) dot = fmaf(qv[i], to_f(k[lane + 32 * i]), dot);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
        const float x = capped_score(dot * s.scale, s), mn = fmaxf(m, x), keep = expf(m - mn), w = expf(x - mn);
        m = mn;
        l = fmaf(l, keep, w);
#pragma unroll
        for (int i = 0; i < NR; ++i)
            if (lane + 32 * i < s.vdim) acc[i] = fmaf(acc[i], keep, w * to_f(v[lane + 32 * i]));
    }
#pragma unroll
    for (int i = 0; i < NR; ++i)
        if (lane + 32 * i < s.v_pad) sm[warp * s.v_pad + lane + 32 * i] = acc[i];
    if (lane == 0) {
        ml[warp][0] = m;
        ml[warp][1] = l;
    }
    __syncthreads();
    float top = ml[0][0];
#pragma unroll
    for (int w = 1; w < kGroupedWarps; ++w) top = fmaxf(top, ml[w][0]);
    float sum = 0.0f, f[kGroupedWarps];
#pragma unroll
    for (int w = 0; w < kGroupedWarps; ++w) {
        f[w] = expf(ml[w][0] - top);
        sum = fmaf(ml[w][1], f[w], sum);
    }
    const T *gate = proj + row * ld + s.off_g + h * s.vdim;
    for (int j = threadIdx.x; j < s.vdim; j += blockDim.x) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kGroupedWarps; ++w) v = fmaf(sm[w * s.v_pad + j], f[w], v);
        out[row * ld_out + h * s.vdim + j] = from_f<T>(v / sum * sigmoid_f(to_f(gate[j])));
    }
}

constexpr int kGroupedTile = 16;     // positions per warp and turn
constexpr int kGroupedValues = 128;  // value columns per block

__host__ __device__ inline int grouped_stage_bytes(int dim_pad, int v_cols) { return kGroupedTile * ((dim_pad + 8) * 2 + (v_cols + 8) * 2); }
__host__ __device__ inline int grouped_smem_bytes(int dim_pad, int v_cols, int stages)
{
    const int ring = kGroupedWarps * stages * grouped_stage_bytes(dim_pad, v_cols), merge = kGroupedWarps * 16 * (v_cols + 4) * 4;
    return 16 * (dim_pad + 8) * 2 + (ring > merge ? ring : merge);
}

// Positions per range: a multiple of the block's turn, the same for all ranges of a row.
__device__ __forceinline__ int grouped_range(int positions, int splits)
{
    constexpr int turn = kGroupedWarps * kGroupedTile;
    return ((positions + turn - 1) / turn + splits - 1) / splits * turn;
}

// bf16: 16 query heads of one key / value head against a range of positions.  Every warp streams tiles of 16 positions of its own through
// a ring of asynchronous copies, scores them, and keeps its own running maximum, sum and weighted values (weights enter the
// second product as the sum of two bf16 values); the warps meet once, at the end.
// part_o [row][heads][splits][v_pad], part_ml [row][heads][splits][2].  VU: value tiles of 8 columns.
// grid: (splits, kv_heads * head tiles * value slices, rows)
template <int VU>
__global__ void __launch_bounds__(kGroupedWarps * 32)
grouped_split_kernel(float *__restrict__ part_o, float *__restrict__ part_ml, const __nv_bfloat16 *__restrict__ proj, long long ld, const GroupedShape s, int stages, int head_tiles,
                     const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int row0)
{
    using namespace mma16;
    extern __shared__ __align__(16) uint8_t grouped_smem[];
    __shared__ float merge_ml[kGroupedWarps][16][2];
    const int share = s.heads / s.kv_heads, slices = (s.v_pad + kGroupedValues - 1) / kGroupedValues;
    const int slice = blockIdx.y % slices, tile = blockIdx.y / slices % head_tiles, g = blockIdx.y / slices / head_tiles;
    const int h0 = g * share + tile * 16, heads = min(16, share - tile * 16);
    const int v0 = slice * kGroupedValues, v_cols = min(kGroupedValues, s.v_pad - v0);
    const int split = blockIdx.x, splits = gridDim.x, local = blockIdx.z, row = row0 + local;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kp = (s.dim_pad + 8) * 2, vp = (v_cols + 8) * 2, stage_bytes = grouped_stage_bytes(s.dim_pad, v_cols);
    const uint32_t q_tile = ptx::smem_u32(grouped_smem), ring = q_tile + 16 * kp + warp * stages * stage_bytes;
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[row_entry[row]];
    const int n = e.pos0 + row - e.row0 + 1;      // visible positions
    const int len = grouped_range(n, splits), first = split * len, end = min(first + len, n);
    if (first >= n) return;                       // nothing for this range: the combining kernel skips it by the same rule
    const __nv_bfloat16 *keys = grouped_cache<__nv_bfloat16>(s, e) + g * s.dim_pad;
    const __nv_bfloat16 *values = grouped_cache<__nv_bfloat16>(s, e) + s.kv_heads * s.dim_pad + g * s.v_pad + v0;
    constexpr int turn = kGroupedWarps * kGroupedTile;
    const int k_pieces = s.dim_pad / 8, v_pieces = v_cols / 8, pieces = k_pieces + v_pieces;
    auto fetch = [&](int t, int b) {
        const uint32_t dst = ring + b * stage_bytes;
        for (int i = lane; i < kGroupedTile * pieces; i += 32) {
            const int r = i / pieces, c = i % pieces;
            const bool key = c < k_pieces;
            const uint32_t at = key ? dst + r * kp + c * 16 : dst + kGroupedTile * kp + r * vp + (c - k_pieces) * 16;
            const __nv_bfloat16 *src = (key ? keys + c * 8 : values + (c - k_pieces) * 8) + static_cast<long long>(t + r) * s.row_pitch;
            if (t + r < end)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(at), "l"(src) : "memory");
            else
                ptx::sts128(at, 0u, 0u, 0u, 0u);
        }
    };
    const int mine = first + warp * kGroupedTile;
    for (int b = 0; b < stages - 1; ++b) {
        if (mine + b * turn < end) fetch(mine + b * turn, b);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int i = threadIdx.x; i < 16 * k_pieces; i += blockDim.x) {
        const int h = i / k_pieces, c = i % k_pieces;
        const uint4 v = h < heads ? *reinterpret_cast<const uint4 *>(proj + row * ld + (h0 + h) * s.dim_pad + c * 8) : make_uint4(0u, 0u, 0u, 0u);
        ptx::sts128(q_tile + h * kp + c * 16, v.x, v.y, v.z, v.w);
    }
    __syncthreads();
    const int r = lane >> 2, c2 = (lane & 3) * 2;
    float m[2] = {-FLT_MAX, -FLT_MAX}, l[2] = {0.0f, 0.0f};
    float O[VU][4] = {};
    for (int t = mine, it = 0; t < end; t += turn, ++it) {
        if (t + (stages - 1) * turn < end) fetch(t + (stages - 1) * turn, (it + stages - 1) % stages);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (stages == 4)
            asm volatile("cp.async.wait_group 3;" ::: "memory");
        else if (stages == 3)
            asm volatile("cp.async.wait_group 2;" ::: "memory");
        else
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncwarp();
        const uint32_t kt = ring + it % stages * stage_bytes, vt = kt + kGroupedTile * kp;
        float sc[2][4] = {};
        for (int k = 0; k < s.dim_pad / 16; ++k) {
            uint32_t a[4], f[4];
            a_frag(a, q_tile, kp, 0, k * 16, lane);
            b_frag(f, kt, kp, 0, k * 16, lane);
            mma(sc[0], a, f[0], f[1]);
            mma(sc[1], a, f[2], f[3]);
        }
        float top[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float x = t + j * 8 + c2 + (i & 1) < end ? capped_score(sc[j][i] * s.scale, s) : -FLT_MAX;
                sc[j][i] = x;
                top[i >> 1] = fmaxf(top[i >> 1], x);
            }
        float f[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], 1));
            top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], 2));
            const float now = fmaxf(m[i], top[i]);   // position t itself is visible: finite
            f[i] = expf(m[i] - now);
            m[i] = now;
            l[i] *= f[i];
        }
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float a = sc[j][2 * i] == -FLT_MAX ? 0.0f : expf(sc[j][2 * i] - m[i]), b = sc[j][2 * i + 1] == -FLT_MAX ? 0.0f : expf(sc[j][2 * i + 1] - m[i]);
                l[i] += a + b;
                split2(a, b, hi[2 * j + i], lo[2 * j + i]);
            }
#pragma unroll
        for (int u = 0; u < VU; u += 2) {
            if (u * 8 >= v_cols) continue;
            uint32_t w[4];
            b_frag_t(w, vt, vp, 0, u * 8, lane);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                O[u + j][0] *= f[0];
                O[u + j][1] *= f[0];
                O[u + j][2] *= f[1];
                O[u + j][3] *= f[1];
                mma(O[u + j], hi, w[2 * j], w[2 * j + 1]);
                mma(O[u + j], lo, w[2 * j], w[2 * j + 1]);
            }
        }
        __syncwarp();   // this stage may be filled again
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    }
    if ((lane & 3) == 0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            merge_ml[warp][r + 8 * i][0] = m[i];
            merge_ml[warp][r + 8 * i][1] = l[i];
        }
    }
    __syncthreads();   // every warp is done with its ring: the merge takes its place
    float *merge = reinterpret_cast<float *>(grouped_smem + 16 * kp);
    const int mp = v_cols + 4;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        float all = merge_ml[0][r + 8 * i][0];
#pragma unroll
        for (int w = 1; w < kGroupedWarps; ++w) all = fmaxf(all, merge_ml[w][r + 8 * i][0]);
        const float f = expf(m[i] - all);
#pragma unroll
        for (int u = 0; u < VU; ++u)
            if (u * 8 < v_cols)
                *reinterpret_cast<float2 *>(merge + (warp * 16 + r + 8 * i) * mp + u * 8 + c2) = make_float2(O[u][2 * i] * f, O[u][2 * i + 1] * f);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < heads * v_cols; i += blockDim.x) {
        const int h = i / v_cols, c = i % v_cols;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kGroupedWarps; ++w) v += merge[(w * 16 + h) * mp + c];
        part_o[((static_cast<long long>(local) * s.heads + h0 + h) * splits + split) * s.v_pad + v0 + c] = v;
    }
    if (slice == 0 && static_cast<int>(threadIdx.x) < heads) {
        const int h = threadIdx.x;
        float all = merge_ml[0][h][0], sum = 0.0f;
#pragma unroll
        for (int w = 1; w < kGroupedWarps; ++w) all = fmaxf(all, merge_ml[w][h][0]);
#pragma unroll
        for (int w = 0; w < kGroupedWarps; ++w) sum += merge_ml[w][h][1] * expf(merge_ml[w][h][0] - all);
        float *ml = part_ml + ((static_cast<long long>(local) * s.heads + h0 + h) * splits + split) * 2;
        ml[0] = all;
        ml[1] = sum;
    }
}

constexpr int kGroupedMaxSplits = 128;

constexpr int kGroupedCombineWarps = 8;

// The ranges of one head put together, the output gate: every warp adds up every eighth range.  grid: (heads, rows)
__global__ void __launch_bounds__(kGroupedCombineWarps * 32)
grouped_combine_kernel(__nv_bfloat16 *__restrict__ out, int ld_out, const float *__restrict__ part_o, const float *__restrict__ part_ml, int splits, const __nv_bfloat16 *__restrict__ proj,
                       long long ld, const GroupedShape s, const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int row0)
{
    extern __shared__ float sm[];   // [warps][v_pad]
    const int h = blockIdx.x, row = row0 + blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[row_entry[row]];
    const int n = e.pos0 + row - e.row0 + 1, len = grouped_range(n, splits), used = (n + len - 1) / len;
    const long long at = (static_cast<long long>(blockIdx.y) * s.heads + h) * splits;
    const float *ml = part_ml + at * 2, *po = part_o + at * s.v_pad;
    float m[kGroupedMaxSplits / 32], l[kGroupedMaxSplits / 32], sum = 0.0f;
#pragma unroll
    for (int i = 0; i < kGroupedMaxSplits / 32; ++i) {
        const float2 x = lane + 32 * i < used ? *reinterpret_cast<const float2 *>(ml + 2 * (lane + 32 * i)) : make_float2(-FLT_MAX, 0.0f);
        m[i] = x.x;
        l[i] = x.y;
    }
    float all = m[0];
#pragma unroll
    for (int i = 1; i < kGroupedMaxSplits / 32; ++i) all = fmaxf(all, m[i]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) all = fmaxf(all, __shfl_xor_sync(0xffffffffu, all, o));
#pragma unroll
    for (int i = 0; i < kGroupedMaxSplits / 32; ++i) sum = fmaf(l[i], expf(m[i] - all), sum);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    for (int c = 4 * lane; c < s.v_pad; c += 128) {
        float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 4
        for (int i = warp; i < used; i += kGroupedCombineWarps) {
            const float4 v = load4(po + static_cast<long long>(i) * s.v_pad + c);
            const float w = expf(ml[2 * i] - all);
            acc.x = fmaf(v.x, w, acc.x); acc.y = fmaf(v.y, w, acc.y); acc.z = fmaf(v.z, w, acc.z); acc.w = fmaf(v.w, w, acc.w);
        }
        store4(sm + warp * s.v_pad + c, acc);
    }
    __syncthreads();
    const __nv_bfloat16 *gate = proj + row * ld + s.off_g + h * s.vdim;
    for (int j = threadIdx.x; j < s.vdim; j += blockDim.x) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kGroupedCombineWarps; ++w) v += sm[w * s.v_pad + j];
        out[static_cast<long long>(row) * ld_out + h * s.vdim + j] = __float2bfloat16_rn(v / sum * sigmoid_f(to_f(gate[j])));
    }
}

}  // namespace dec
}  // namespace gptb200
