// Products of up to eight rows with a bf16 weight matrix stored [n][k]: out[m][n] = x[m][k] . w[n][k], fp32 accumulation, with the
// outputs of the bf16 tensor-core form (OutKind).  The weights are streamed once: a warp takes two weight rows at a time, 512
// contiguous bytes of each per step, the activations come from shared memory.
//
// The kernel may be launched with programmatic stream serialization: it requests its first weights while its predecessor on
// the stream still runs and touches activations and outputs only after griddepcontrol.wait (weights are never written
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
};

constexpr int kGemvThreads = 256;
constexpr int kGemvUnroll = 4;   // 16-byte loads in flight per lane and weight row

__device__ __forceinline__ float bf16_round_store(uint16_t *dst, float v)
{
    const uint32_t w = ptx::pack_bf16x2(v, v);
    *dst = static_cast<uint16_t>(w & 0xFFFFu);
    return v;
}

// One finished value (OUT_GLU: `v` is the gate and `u` the up column of the pair).
__device__ __forceinline__ void gemv_emit(const GemvParams &p, int m, int n, float v, float u)
{
    if (p.out_kind == OUT_F32) {
        static_cast<float *>(p.out)[m * p.ldo + n] = v;
    } else if (p.out_kind == OUT_BF16) {
        if (n >= p.tail_col)
            p.tail[static_cast<long long>(m) * p.tail_pitch + (n - p.tail_col)] = v;
        else
            bf16_round_store(static_cast<uint16_t *>(p.out) + m * p.ldo + n, v);
    } else if (p.out_kind == OUT_GLU) {
        bf16_round_store(static_cast<uint16_t *>(p.out) + m * p.ldo + (n >> 6) * 32 + (n & 31), gelu_tanh(v) * u);
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
    if (out_kind == OUT_GLU) {
        ra = (i >> 5) * 64 + (i & 31);
        rb = ra + 32;
    } else {
        ra = 2 * i;
        rb = 2 * i + 1;
    }
}

template <int MR>
__global__ void __launch_bounds__(kGemvThreads)
gemv_bf16_kernel(const GemvParams p)
{
    extern __shared__ uint4 gemv_x[];   // [MR][K / 8]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int chunks = p.K >> 3;
    const int pairs = p.out_kind == OUT_GLU ? p.N / 2 : (p.N + 1) / 2;
    const int stride = gridDim.x * (kGemvThreads / 32);
    int pair = blockIdx.x * (kGemvThreads / 32) + warp;

    uint4 wa[kGemvUnroll], wb[kGemvUnroll];
    auto fetch = [&](int i, int c0) {
        int ra, rb;
        gemv_pair(i, p.out_kind, ra, rb);
        const uint4 *a = reinterpret_cast<const uint4 *>(p.w + static_cast<long long>(ra) * p.K);
        const uint4 *b = reinterpret_cast<const uint4 *>(p.w + static_cast<long long>(rb) * p.K);
#pragma unroll
        for (int u = 0; u < kGemvUnroll; ++u) {
            const int c = c0 + u * 32 + lane;
            wa[u] = c < chunks ? __ldg(a + c) : make_uint4(0u, 0u, 0u, 0u);
            wb[u] = c < chunks && rb < p.N ? __ldg(b + c) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    if (pair < pairs) fetch(pair, 0);
    grid_dependency_wait();
    grid_dependency_launch();
    for (int i = threadIdx.x; i < MR * chunks; i += kGemvThreads) {
        const int m = i / chunks, c = i % chunks;
        gemv_x[i] = m < p.M ? *(reinterpret_cast<const uint4 *>(p.x + m * p.ldx) + c) : make_uint4(0u, 0u, 0u, 0u);
    }
    __syncthreads();
    for (; pair < pairs; pair += stride) {
        float sa[MR], sb[MR];
#pragma unroll
        for (int m = 0; m < MR; ++m) sa[m] = sb[m] = 0.0f;
        for (int c0 = 0; c0 < chunks; c0 += 32 * kGemvUnroll) {
            if (c0 > 0) fetch(pair, c0);
#pragma unroll
            for (int u = 0; u < kGemvUnroll; ++u) {
                const int c = c0 + u * 32 + lane;
                if (c < chunks) {
#pragma unroll
                    for (int m = 0; m < MR; ++m) {
                        const uint4 xv = gemv_x[m * chunks + c];
                        sa[m] = dot8(wa[u], xv, sa[m]);
                        sb[m] = dot8(wb[u], xv, sb[m]);
                    }
                }
            }
        }
        const int done = pair;
        if (pair + stride < pairs) fetch(pair + stride, 0);   // the next pair's first weights travel during the reduction
        int ra, rb;
        gemv_pair(done, p.out_kind, ra, rb);
#pragma unroll
        for (int m = 0; m < MR; ++m) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                sa[m] += __shfl_xor_sync(0xffffffffu, sa[m], o);
                sb[m] += __shfl_xor_sync(0xffffffffu, sb[m], o);
            }
        }
#pragma unroll
        for (int m = 0; m < MR; ++m) {
            if (m < p.M && lane == m) {
                gemv_emit(p, m, ra, sa[m], sb[m]);
                if (p.out_kind != OUT_GLU && rb < p.N) gemv_emit(p, m, rb, sb[m], 0.0f);
            }
        }
    }
}

}  // namespace gptb200
