// Products of up to eight rows with a bf16 weight matrix stored [n][k]: out[m][n] = x[m][k] . w[n][k], fp32 accumulation, with the
// outputs of the bf16 tensor-core form (OutKind).  The weights are streamed once and the activations come from shared memory.
// One row: a warp takes two weight rows at a time, 512 contiguous bytes of each per step, fp32 FMAs.  Two to eight rows:
// gemv_bf16_mma_kernel.
//
// The kernels may be launched with programmatic stream serialization: they request their first weights while their predecessor on
// the stream still runs and touch activations and outputs only after griddepcontrol.wait (weights are never written
// by a kernel of a step).
#pragma once

#include "gemm_sm100.cuh"

namespace gptb200 {

__device__ __forceinline__ void grid_dependency_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void grid_dependency_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

struct GemvParams {
    int M, N, K;            // K in elements, a multiple of 8
    const uint16_t *x;      // bf16 [M][ldx]
    long long ldx;
    const uint16_t *w;      // bf16 [N][K]
    int out_kind;           // OutKind
    void *out;
    long long ldo;          // elements of the output type
    float *tail;
    int tail_col, tail_pitch;
    const uint16_t *factor;
    const int *factor_rows;
    int factor_pitch;
    const float *bias;      // null: none
    int silu_cols;          // OUT_BF16: silu is applied to the columns before this one
    int group_cols;         // columns per group (a multiple of 64; >= N: one group); blockIdx.y counts the groups,
    long long group_x;      //   whose rows of x lie this many elements apart
    int k_warps;            // one row: warps of a block that share a pair of weight rows (1, 2, 4, 8)
};

constexpr int kGemvThreads = 256;
constexpr int kGemvUnroll = 4;   // 16-byte loads in flight per lane and weight row

__device__ __forceinline__ float bf16_round_store(uint16_t *dst, float v)
{
    const uint32_t w = ptx::pack_bf16x2(v, v);
    *dst = static_cast<uint16_t>(w & 0xFFFFu);
    return v;
}

// One finished value (gated kinds: `v` is the gate and `u` the up column of the pair).
__device__ __forceinline__ void gemv_emit(const GemvParams &p, int m, int n, float v, float u)
{
    if (p.bias) {
        v += __ldg(p.bias + n);
        if (is_glu(p.out_kind)) u += __ldg(p.bias + n + 32);
    }
    if (p.out_kind == OUT_F32) {
        static_cast<float *>(p.out)[m * p.ldo + n] = v;
    } else if (p.out_kind == OUT_BF16) {
        if (n >= p.tail_col)
            p.tail[static_cast<long long>(m) * p.tail_pitch + (n - p.tail_col)] = v;
        else
            bf16_round_store(static_cast<uint16_t *>(p.out) + m * p.ldo + n, n < p.silu_cols ? silu_fast(v) : v);
    } else if (is_glu(p.out_kind)) {
        bf16_round_store(static_cast<uint16_t *>(p.out) + m * p.ldo + (n >> 6) * 32 + (n & 31), (p.out_kind == OUT_GLU ? gelu_tanh(v) : silu_fast(v)) * u);
    } else {
        const float f = __uint_as_float(static_cast<uint32_t>(p.factor[static_cast<long long>(p.factor_rows[m]) * p.factor_pitch + n]) << 16);
        bf16_round_store(static_cast<uint16_t *>(p.out) + m * p.ldo + n, gelu_tanh(v) * f);
    }
}

__device__ __forceinline__ float dot8(const uint4 &a, const uint4 &b, float acc)
{
    const uint32_t x[4] = {a.x, a.y, a.z, a.w}, y[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        acc = fmaf(bf16_lo(x[e]), bf16_lo(y[e]), acc);
        acc = fmaf(bf16_hi(x[e]), bf16_hi(y[e]), acc);
    }
    return acc;
}

// The two weight rows of pair `i`: adjacent rows, or a gate row and its up row (groups of 32 gate | 32 up).
__device__ __forceinline__ void gemv_pair(int i, int out_kind, int &ra, int &rb)
{
    if (is_glu(out_kind)) {
        ra = (i >> 5) * 64 + (i & 31);
        rb = ra + 32;
    } else {
        ra = 2 * i;
        rb = 2 * i + 1;
    }
}

// SHARED: p.k_warps warps share a pair of weight rows and every warp has at most one pair.
template <bool SHARED>
__global__ void __launch_bounds__(kGemvThreads)
gemv_bf16_kernel(const GemvParams p)
{
    extern __shared__ uint4 gemv_x[];   // [K / 8]
    __shared__ float2 parts[SHARED ? kGemvThreads / 32 : 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int chunks = p.K >> 3;
    const int n0 = blockIdx.y * p.group_cols, N = min(p.N - n0, p.group_cols);   // this group's columns
    const uint16_t *w = p.w + static_cast<long long>(n0) * p.K, *x = p.x + blockIdx.y * p.group_x;
    const int pairs = is_glu(p.out_kind) ? N / 2 : (N + 1) / 2;
    const int k_warps = SHARED ? p.k_warps : 1;
    const int per_block = (kGemvThreads / 32) / k_warps, stride = gridDim.x * per_block;
    int pair = blockIdx.x * per_block + warp / k_warps;
    // this warp's share of k, in chunks of 8
    const int share = (chunks + k_warps - 1) / k_warps, begin = SHARED ? (warp % k_warps) * share : 0, end = SHARED ? min(chunks, begin + share) : chunks;

    uint4 wa[kGemvUnroll], wb[kGemvUnroll];
    auto fetch = [&](int i, int c0) {
        int ra, rb;
        gemv_pair(i, p.out_kind, ra, rb);
        const uint4 *a = reinterpret_cast<const uint4 *>(w + static_cast<long long>(ra) * p.K);
        const uint4 *b = reinterpret_cast<const uint4 *>(w + static_cast<long long>(rb) * p.K);
#pragma unroll
        for (int u = 0; u < kGemvUnroll; ++u) {
            const int c = c0 + u * 32 + lane;
            wa[u] = c < end ? __ldg(a + c) : make_uint4(0u, 0u, 0u, 0u);
            wb[u] = c < end && rb < N ? __ldg(b + c) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    if (pair < pairs) fetch(pair, begin);
    grid_dependency_wait();
    grid_dependency_launch();
    for (int i = threadIdx.x; i < chunks; i += kGemvThreads) gemv_x[i] = *(reinterpret_cast<const uint4 *>(x) + i);
    __syncthreads();
    for (; pair < pairs; pair += stride) {
        float sa = 0.0f, sb = 0.0f;
        for (int c0 = begin; c0 < end; c0 += 32 * kGemvUnroll) {
            if (c0 > begin) fetch(pair, c0);
#pragma unroll
            for (int u = 0; u < kGemvUnroll; ++u) {
                const int c = c0 + u * 32 + lane;
                if (c < end) {
                    const uint4 xv = gemv_x[c];
                    sa = dot8(wa[u], xv, sa);
                    sb = dot8(wb[u], xv, sb);
                }
            }
        }
        const int done = pair;
        if (pair + stride < pairs) fetch(pair + stride, begin);   // the next pair's first weights travel during the reduction
        int ra, rb;
        gemv_pair(done, p.out_kind, ra, rb);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            sa += __shfl_xor_sync(0xffffffffu, sa, o);
            sb += __shfl_xor_sync(0xffffffffu, sb, o);
        }
        if (SHARED) {
            if (lane == 0) parts[warp] = make_float2(sa, sb);
            continue;
        }
        if (lane == 0) {
            gemv_emit(p, 0, n0 + ra, sa, sb);
            if (!is_glu(p.out_kind) && rb < N) gemv_emit(p, 0, n0 + rb, sb, 0.0f);
        }
    }
    if (SHARED) {
        __syncthreads();
        const int done = blockIdx.x * per_block + static_cast<int>(threadIdx.x);
        if (static_cast<int>(threadIdx.x) < per_block && done < pairs) {
            float sa = 0.0f, sb = 0.0f;
            for (int i = 0; i < k_warps; ++i) {
                sa += parts[threadIdx.x * k_warps + i].x;
                sb += parts[threadIdx.x * k_warps + i].y;
            }
            int ra, rb;
            gemv_pair(done, p.out_kind, ra, rb);
            gemv_emit(p, 0, n0 + ra, sa, sb);
            if (!is_glu(p.out_kind) && rb < N) gemv_emit(p, 0, n0 + rb, sb, 0.0f);
        }
    }
}

// Two to eight rows: the same stream of weights as the A operand of m16n8k16 products (16 weight rows, up to eight rows of x).  A
// block takes TILES x 16 weight rows (gated kinds: 16 gate rows and their 16 up rows) and its eight warps share k, so no value of x is read
// twice by a block and x comes straight from L2.  The order of k inside a block
// of 32 is permuted alike on both sides so that a lane loads 16 contiguous bytes of a row: piece c of a block (8 values) feeds
// two products, values 0-3 the first and 4-7 the second.
constexpr int kGemvMmaUnroll = 4;   // blocks of 32 k in flight per warp

__device__ __forceinline__ void gemv_mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int TILES>
__global__ void __launch_bounds__(kGemvThreads)
gemv_bf16_mma_kernel(const GemvParams p)
{
    __shared__ float sums[8 * TILES * 16 * 8];   // [warp][weight row][row of x]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c = lane & 3;
    const int n0 = blockIdx.y * p.group_cols, N = min(p.N - n0, p.group_cols);   // this group's columns
    const uint16_t *w = p.w + static_cast<long long>(n0) * p.K;
    // weight rows of the block's tiles
    int row[TILES];
#pragma unroll
    for (int t = 0; t < TILES; ++t)
        row[t] = is_glu(p.out_kind) ? (blockIdx.x >> 1) * 64 + (blockIdx.x & 1) * 16 + t * 32 : (blockIdx.x * TILES + t) * 16;
    const int blocks = (p.K + 31) / 32, per_warp = (blocks + 7) / 8;
    const int first = warp * per_warp, end = min(blocks, first + per_warp);
    uint4 wv[kGemvMmaUnroll][TILES][2];
    auto fetch = [&](int blk) {
#pragma unroll
        for (int u = 0; u < kGemvMmaUnroll; ++u) {
            const int k = (blk + u) * 32 + c * 8;
#pragma unroll
            for (int t = 0; t < TILES; ++t)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int r = row[t] + g + 8 * half;
                    wv[u][t][half] = blk + u < end && k < p.K && r < N ? __ldg(reinterpret_cast<const uint4 *>(w + static_cast<long long>(r) * p.K + k)) : make_uint4(0u, 0u, 0u, 0u);
                }
        }
    };
    fetch(first);
    grid_dependency_wait();
    grid_dependency_launch();
    float acc[TILES][4] = {};
    const bool live = g < p.M;   // this lane's row of x
    const uint16_t *xs = p.x + blockIdx.y * p.group_x + (live ? g : 0) * p.ldx + c * 8;
    for (int blk = first; blk < end; blk += kGemvMmaUnroll) {
        if (blk > first) fetch(blk);
        uint4 xv[kGemvMmaUnroll];
#pragma unroll
        for (int u = 0; u < kGemvMmaUnroll; ++u)
            xv[u] = live && blk + u < end && (blk + u) * 32 + c * 8 < p.K ? *reinterpret_cast<const uint4 *>(xs + (blk + u) * 32) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
        for (int u = 0; u < kGemvMmaUnroll; ++u) {
            const uint4 x = xv[u];
#pragma unroll
            for (int t = 0; t < TILES; ++t) {
                const uint4 a = wv[u][t][0], b = wv[u][t][1];
                gemv_mma_bf16(acc[t], a.x, b.x, a.y, b.y, x.x, x.y);
                gemv_mma_bf16(acc[t], a.z, b.z, a.w, b.w, x.z, x.w);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < TILES; ++t)
#pragma unroll
        for (int i = 0; i < 4; ++i) sums[(warp * TILES * 16 + t * 16 + g + (i >> 1) * 8) * 8 + 2 * c + (i & 1)] = acc[t][i];
    __syncthreads();
    const int outputs = is_glu(p.out_kind) ? 128 : TILES * 128;
    for (int i = threadIdx.x; i < outputs; i += kGemvThreads) {
        const int r = i >> 3, m = i & 7;
        if (m >= p.M) continue;
        float v = 0.0f, up = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            v += sums[(w * TILES * 16 + r) * 8 + m];
            if (TILES == 2 && is_glu(p.out_kind)) up += sums[(w * TILES * 16 + 16 + r) * 8 + m];
        }
        const int n = is_glu(p.out_kind) ? row[0] + r : blockIdx.x * TILES * 16 + r;
        if (n < N) gemv_emit(p, m, n0 + n, v, up);
    }
}

}  // namespace gptb200
