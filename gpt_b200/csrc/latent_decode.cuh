// Latent attention of a few rows (decoding, short portions) in bf16: the absorbed form in three launches, so that the cached
// rows -- the only thing whose size grows -- are streamed once for all heads.
//
//   latent_query_kernel    q_u mapped into the latent space and the rotated query part, fp32; one more block per row norms the
//                          row's own latent, rotates its key part and appends both to the cache
//   latent_split_kernel    one block per (row, 16 heads, range of positions): tiles of 32 cached rows serve as keys AND as values from
//                          one copy in shared memory; queries and softmax weights enter the products as sums of two bf16 values;
//                          running maximum and sum per head; the range's weighted latent goes to scratch
//   latent_combine_kernel  the ranges of one head put together, W_uv, the output gate
#pragma once

#include "latent_attention.cuh"
#include "mamba2_chunk.cuh"   // mma16

namespace gptb200 {
namespace dec {

constexpr int kQuerySlice = 64;   // latent columns per block of the query kernel

// q_out [row][heads][row_pitch]: scaled query in the cached rows' space.  grid: (heads * slices + own_keys, rows)
__global__ void __launch_bounds__(256)
latent_query_kernel(float *__restrict__ q_out, const __nv_bfloat16 *__restrict__ proj, long long ld, const __nv_bfloat16 *__restrict__ w_uk, const float2 *__restrict__ table,
                    const float *__restrict__ norm_w, float eps, const LatentShape s, const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int row0)
{
    __shared__ float part[32][kQuerySlice];
    __shared__ float qs[1024];
    __shared__ float red[32];
    const int slices = (s.rank_pitch + kQuerySlice - 1) / kQuerySlice;
    const int row = row0 + blockIdx.y;
    const int h = blockIdx.x / slices, c0 = (blockIdx.x % slices) * kQuerySlice;
    const int tid = threadIdx.x;
    // this block's first weights travel while the kernel before still runs
    const int cg = (tid & 7) * 8, dg = tid >> 3;
    const bool mapper = h < s.heads;
    const bool col_ok = mapper && c0 + cg < s.rank_pitch;
    const __nv_bfloat16 *w = w_uk + static_cast<long long>(h) * s.dim_pad * s.rank_pitch + c0 + cg;
    uint4 w0[4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
        w0[i] = col_ok && dg + 32 * i < s.dim ? __ldg(reinterpret_cast<const uint4 *>(w + static_cast<long long>(dg + 32 * i) * s.rank_pitch)) : make_uint4(0u, 0u, 0u, 0u);
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[row_entry[row]];
    const __nv_bfloat16 *r = proj + row * ld;
    const float2 *cs = table + static_cast<long long>(row) * s.rot_half;
    if (!mapper) {
        const __nv_bfloat16 *d = r + s.off_dkv;
        __nv_bfloat16 *dst = latent_cache<__nv_bfloat16>(s, e) + static_cast<long long>(e.pos0 + row - e.row0) * s.row_pitch;
        float ss = 0.0f;
        for (int i = tid; i < s.kv_rank; i += blockDim.x) {
            const float v = to_f(d[i]);
            ss = fmaf(v, v, ss);
        }
        const float inv = rsqrtf(block_sum(ss, red) / s.kv_rank + eps);
        for (int i = tid; i < s.rank_pitch; i += blockDim.x) dst[i] = __float2bfloat16_rn(i < s.kv_rank ? to_f(d[i]) * inv * norm_w[i] : 0.0f);
        for (int k = tid; k < s.row_pitch - s.rank_pitch; k += blockDim.x) dst[s.rank_pitch + k] = __float2bfloat16_rn(rotated(d + s.kv_rank, k, cs, s));
        return;
    }
    const __nv_bfloat16 *q = r + h * s.q_stride;
    float *out = q_out + (static_cast<long long>(blockIdx.y) * s.heads + h) * s.row_pitch;
    for (int d = tid; d < s.dim; d += blockDim.x) qs[d] = to_f(q[d]);
    if (c0 == 0)
        for (int k = tid; k < s.row_pitch - s.rank_pitch; k += blockDim.x) out[s.rank_pitch + k] = rotated(q + s.dim_pad, k, cs, s) * s.scale;
    __syncthreads();
    float acc[8] = {};
    auto add = [&](const uint4 &v, float x) {
        const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            acc[2 * i] = fmaf(x, bf16_lo(u[i]), acc[2 * i]);
            acc[2 * i + 1] = fmaf(x, bf16_hi(u[i]), acc[2 * i + 1]);
        }
    };
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (dg + 32 * i < s.dim) add(w0[i], qs[dg + 32 * i]);
    if (col_ok)
        for (int d = dg + 128; d < s.dim; d += 32) add(__ldg(reinterpret_cast<const uint4 *>(w + static_cast<long long>(d) * s.rank_pitch)), qs[d]);
#pragma unroll
    for (int i = 0; i < 8; ++i) part[dg][cg + i] = acc[i];
    __syncthreads();
    if (tid < kQuerySlice && c0 + tid < s.rank_pitch) {
        float v = 0.0f;
#pragma unroll
        for (int i = 0; i < 32; ++i) v += part[i][tid];
        out[c0 + tid] = v * s.scale;
    }
}

constexpr int kSplitTile = 32;       // positions per tile
constexpr int kSplitThreads = 256;
constexpr int kSplitUnits = 6;       // 16-column units of the latent per warp (rank_pitch <= 768)

__host__ __device__ inline int split_smem_bytes(int row_pitch)
{
    const int pitch = (row_pitch + 8) * 2;
    return 2 * 16 * pitch + 2 * kSplitTile * pitch + 2 * 16 * (kSplitTile + 1) * 4 + 2 * 16 * (kSplitTile + 8) * 2 + 3 * 16 * 4;
}

// Positions per range: a multiple of the tile, the same for all ranges of a row.
__device__ __forceinline__ int split_length(int positions, int splits)
{
    const int tiles = (positions + kSplitTile - 1) / kSplitTile;
    return (tiles + splits - 1) / splits * kSplitTile;
}

// part_o [row][heads][splits][rank_pitch], part_ml [row][heads][splits][2].  grid: (splits, head groups of 16, rows)
__global__ void __launch_bounds__(kSplitThreads)
latent_split_kernel(float *__restrict__ part_o, float *__restrict__ part_ml, const float *__restrict__ q_in, const LatentShape s, const StepEntry *__restrict__ entries,
                    const int *__restrict__ row_entry, int row0)
{
    using namespace mma16;
    extern __shared__ __align__(16) uint8_t split_smem[];
    const int pitch = (s.row_pitch + 8) * 2;
    const uint32_t base = ptx::smem_u32(split_smem);
    const uint32_t q_hi = base, q_lo = q_hi + 16 * pitch, tiles = q_lo + 16 * pitch;
    float *sc = reinterpret_cast<float *>(split_smem + 32 * pitch + 2 * kSplitTile * pitch);   // [2][16][tile + 1]
    const int p_pitch = (kSplitTile + 8) * 2;
    const uint32_t p_hi = tiles + 2 * kSplitTile * pitch + 2 * 16 * (kSplitTile + 1) * 4, p_lo = p_hi + 16 * p_pitch;
    float *row_m = reinterpret_cast<float *>(split_smem + 32 * pitch + 2 * kSplitTile * pitch + 2 * 16 * (kSplitTile + 1) * 4 + 2 * 16 * p_pitch), *row_l = row_m + 16, *row_f = row_l + 16;
    grid_dependency_wait();
    grid_dependency_launch();
    const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * 16, local = blockIdx.z, row = row0 + local;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int heads = min(16, s.heads - h0);
    const StepEntry e = entries[row_entry[row]];
    const int n = e.pos0 + row - e.row0 + 1;      // visible positions
    const int len = split_length(n, splits), first = split * len, end = min(first + len, n);
    if (first >= n) {                              // nothing for this range: the combining kernel skips it by the same rule
        return;
    }
    const __nv_bfloat16 *cache = latent_cache<__nv_bfloat16>(s, e);
    const int pieces = s.row_pitch / 8;
    auto fetch = [&](int t, int b) {
        for (int i = tid; i < kSplitTile * pieces; i += kSplitThreads) {
            const int r = i / pieces, c = i % pieces;
            const uint32_t dst = tiles + b * kSplitTile * pitch + r * pitch + c * 16;
            if (t + r < end)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(cache + static_cast<long long>(t + r) * s.row_pitch + c * 8) : "memory");
            else
                ptx::sts128(dst, 0u, 0u, 0u, 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(first, 0);
    for (int i = tid; i < 16 * (s.row_pitch / 2); i += kSplitThreads) {
        const int h = i / (s.row_pitch / 2), c = i % (s.row_pitch / 2);
        float2 v = make_float2(0.0f, 0.0f);
        if (h < heads) v = *reinterpret_cast<const float2 *>(q_in + (static_cast<long long>(local) * s.heads + h0 + h) * s.row_pitch + 2 * c);
        uint32_t hi, lo;
        split2(v.x, v.y, hi, lo);
        asm volatile("st.shared.b32 [%0], %1;" ::"r"(q_hi + h * pitch + c * 4), "r"(hi) : "memory");
        asm volatile("st.shared.b32 [%0], %1;" ::"r"(q_lo + h * pitch + c * 4), "r"(lo) : "memory");
    }
    if (tid < 16) {
        row_m[tid] = -FLT_MAX;
        row_l[tid] = 0.0f;
    }
    const int r = lane >> 2, c2 = (lane & 3) * 2;
    const int k_steps = s.row_pitch / 16;
    const int units = s.rank_pitch / 16;
    float O[kSplitUnits][2][4] = {};
    for (int t = first, it = 0; t < end; t += kSplitTile, ++it) {
        const int b = it & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t + kSplitTile < end) fetch(t + kSplitTile, b ^ 1);
        const uint32_t tile = tiles + b * kSplitTile * pitch;
        // scores of 16 positions by a quarter of the inner dimension each: warps 0-1, 2-3, ... share positions
        {
            const int half = warp & 1, kq = warp >> 1;        // positions 16 half .., quarter kq of the k-steps
            const int k0 = kq * ((k_steps + 3) / 4), k1 = min(k_steps, k0 + (k_steps + 3) / 4);
            float a0[4] = {}, a1[4] = {};
            for (int k = k0; k < k1; ++k) {
                uint32_t ah[4], al[4], f[4];
                a_frag(ah, q_hi, pitch, 0, k * 16, lane);
                a_frag(al, q_lo, pitch, 0, k * 16, lane);
                b_frag(f, tile, pitch, half * 16, k * 16, lane);
                mma(a0, ah, f[0], f[1]);
                mma(a0, al, f[0], f[1]);
                mma(a1, ah, f[2], f[3]);
                mma(a1, al, f[2], f[3]);
            }
            // quarters are added in two steps through shared memory, in a fixed order
            float *dst = sc + (kq & 1) * 16 * (kSplitTile + 1);
            auto put = [&](bool add) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int at = (r + (i >> 1) * 8) * (kSplitTile + 1) + half * 16 + c2 + (i & 1);
                    dst[at] = add ? dst[at] + a0[i] : a0[i];
                    dst[at + 8] = add ? dst[at + 8] + a1[i] : a1[i];
                }
            };
            if (kq < 2) put(false);
            __syncthreads();
            if (kq >= 2) put(true);
        }
        __syncthreads();
        {   // 16 threads per head, two positions each
            const int h = tid >> 4, j = (tid & 15) * 2;
            const float *s0 = sc + h * (kSplitTile + 1), *s1 = s0 + 16 * (kSplitTile + 1);
            const float x0 = t + j < end ? s0[j] + s1[j] : -FLT_MAX, x1 = t + j + 1 < end ? s0[j + 1] + s1[j + 1] : -FLT_MAX;
            float top = fmaxf(x0, x1);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
            const float old = row_m[h], m = fmaxf(old, top);
            const float p0 = t + j < end ? expf(x0 - m) : 0.0f, p1 = t + j + 1 < end ? expf(x1 - m) : 0.0f;
            float sum = p0 + p1;
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            uint32_t hi, lo;
            split2(p0, p1, hi, lo);
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_hi + h * p_pitch + j * 2), "r"(hi) : "memory");
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_lo + h * p_pitch + j * 2), "r"(lo) : "memory");
            __syncwarp();   // both heads of the warp have read their old maximum
            if ((tid & 15) == 0) {
                const float f = expf(old - m);
                row_f[h] = f;
                row_m[h] = m;
                row_l[h] = fmaf(row_l[h], f, sum);
            }
        }
        __syncthreads();
        const float fa = row_f[r], fb = row_f[r + 8];
        uint32_t ah[2][4], al[2][4];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            a_frag(ah[k], p_hi, p_pitch, 0, k * 16, lane);
            a_frag(al[k], p_lo, p_pitch, 0, k * 16, lane);
        }
#pragma unroll
        for (int u = 0; u < kSplitUnits; ++u) {
            const int col = (u * 8 + warp) * 16;
            if (u * 8 + warp >= units) continue;
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                O[u][q][0] *= fa;
                O[u][q][1] *= fa;
                O[u][q][2] *= fb;
                O[u][q][3] *= fb;
            }
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                uint32_t f[4];
                b_frag_t(f, tile, pitch, k * 16, col, lane);
                mma(O[u][0], ah[k], f[0], f[1]);
                mma(O[u][0], al[k], f[0], f[1]);
                mma(O[u][1], ah[k], f[2], f[3]);
                mma(O[u][1], al[k], f[2], f[3]);
            }
        }
    }
#pragma unroll
    for (int u = 0; u < kSplitUnits; ++u) {
        if (u * 8 + warp >= units) continue;
        const int col = (u * 8 + warp) * 16;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = r + 8 * i;
            if (h >= heads) continue;
            float *dst = part_o + ((static_cast<long long>(local) * s.heads + h0 + h) * splits + split) * s.rank_pitch + col + c2;
            *reinterpret_cast<float2 *>(dst) = make_float2(O[u][0][2 * i], O[u][0][2 * i + 1]);
            *reinterpret_cast<float2 *>(dst + 8) = make_float2(O[u][1][2 * i], O[u][1][2 * i + 1]);
        }
    }
    if (tid < heads) {
        float *ml = part_ml + ((static_cast<long long>(local) * s.heads + h0 + tid) * splits + split) * 2;
        ml[0] = row_m[tid];
        ml[1] = row_l[tid];
    }
}

constexpr int kCombineRows = 32;   // value rows of W_uv per block

// grid: (heads * value slices, rows)
__global__ void __launch_bounds__(256)
latent_combine_kernel(__nv_bfloat16 *__restrict__ out, int ld_out, const float *__restrict__ part_o, const float *__restrict__ part_ml, int splits, const __nv_bfloat16 *__restrict__ proj,
                      long long ld, const __nv_bfloat16 *__restrict__ w_uv, const LatentShape s, const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int row0)
{
    extern __shared__ float latent[];   // [rank_pitch]
    __shared__ float weight[256];
    __shared__ float total;
    const int slices = (s.vdim + kCombineRows - 1) / kCombineRows;
    const int h = blockIdx.x / slices, v0 = (blockIdx.x % slices) * kCombineRows, row = row0 + blockIdx.y;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[row_entry[row]];
    const int n = e.pos0 + row - e.row0 + 1;
    const int used = (n + split_length(n, splits) - 1) / split_length(n, splits);
    const float *ml = part_ml + (static_cast<long long>(blockIdx.y) * s.heads + h) * splits * 2;
    if (warp == 0) {
        float top = -FLT_MAX, sum = 0.0f;
        for (int i = lane; i < used; i += 32) top = fmaxf(top, ml[2 * i]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
        for (int i = lane; i < used; i += 32) {
            const float f = expf(ml[2 * i] - top);
            weight[i] = f;
            sum = fmaf(ml[2 * i + 1], f, sum);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (lane == 0) total = sum;
    }
    __syncthreads();
    const float *po = part_o + (static_cast<long long>(blockIdx.y) * s.heads + h) * splits * s.rank_pitch;
    for (int j = tid; j < s.rank_pitch; j += blockDim.x) {
        float v = 0.0f;
#pragma unroll 8
        for (int i = 0; i < used; ++i) v = fmaf(po[static_cast<long long>(i) * s.rank_pitch + j], weight[i], v);
        latent[j] = v / total;
    }
    __syncthreads();
    for (int v = v0 + warp; v < min(v0 + kCombineRows, s.vdim); v += 8) {
        const __nv_bfloat16 *w = w_uv + (static_cast<long long>(h) * s.v_pad + v) * s.rank_pitch;
        float acc = 0.0f;
        for (int j = lane * 8; j < s.rank_pitch; j += 256) {
            const uint4 x = __ldg(reinterpret_cast<const uint4 *>(w + j));
            const uint32_t u[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) acc = fmaf(bf16_lo(u[i]), latent[j + 2 * i], fmaf(bf16_hi(u[i]), latent[j + 2 * i + 1], acc));
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) out[static_cast<long long>(row) * ld_out + h * s.vdim + v] = __float2bfloat16_rn(acc * sigmoid_f(to_f(proj[row * ld + s.off_g + h * s.vdim + v])));
    }
}

}  // namespace dec
}  // namespace gptb200
