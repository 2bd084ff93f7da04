// Mamba-2 recurrence over prompts: the state-space duality form in chunks of 64 tokens, on tensor cores.
//
// With a_t the running sum of log-decays inside a chunk and S the state before it,
//   y_t = exp(a_t) C_t S + sum_{s <= t} exp(a_t - a_s) dt_s (C_t . B_s) x_s + D x_t
//   S  <- exp(a_end) S + sum_s exp(a_end - a_s) dt_s B_s x_s^T
// One block carries one head's state for 32 of its value columns through all chunks of a request: S stays in the fp32 accumulators of
// the warps from chunk to chunk, nothing is exchanged through memory, and the next chunk's x, B and C arrive while this
// one is computed.  x, B and C are bf16 as the convolution left them; everything that is fp32 by nature (weights with decays and
// steps, the scaled x, the state) enters a product as the sum of two bf16 values.
#pragma once

#include "mamba2.cuh"

namespace gptb200 {
namespace dec {

constexpr int kChunk = 64;
constexpr int kChunkCols = 32;       // value columns per block
constexpr int kChunkThreads = 128;
constexpr int kChunkMaxState = 128;

namespace mma16 {

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Fragments from a row-major tile in shared memory (pitch in bytes), 16 x 16 at (row, col):
//   a_frag     A operand, M = rows, K = columns
//   a_frag_t   A operand, M = columns, K = rows
//   b_frag     two B operands, N = rows (r[0], r[1]: rows 0-7; r[2], r[3]: rows 8-15), K = columns
//   b_frag_t   two B operands, N = columns (r[0], r[1]: columns 0-7; r[2], r[3]: 8-15), K = rows
__device__ __forceinline__ void a_frag(uint32_t (&r)[4], uint32_t tile, int pitch, int row, int col, int lane)
{
    ldsm4(r, tile + (row + (lane & 15)) * pitch + (col + ((lane >> 4) << 3)) * 2);
}
__device__ __forceinline__ void a_frag_t(uint32_t (&r)[4], uint32_t tile, int pitch, int row, int col, int lane)
{
    ldsm4t(r, tile + (row + (lane & 7) + ((lane >> 4) << 3)) * pitch + (col + (((lane >> 3) & 1) << 3)) * 2);
}
__device__ __forceinline__ void b_frag(uint32_t (&r)[4], uint32_t tile, int pitch, int row, int col, int lane)
{
    ldsm4(r, tile + (row + (lane & 7) + ((lane >> 4) << 3)) * pitch + (col + (((lane >> 3) & 1) << 3)) * 2);
}
__device__ __forceinline__ void b_frag_t(uint32_t (&r)[4], uint32_t tile, int pitch, int row, int col, int lane)
{
    ldsm4t(r, tile + (row + (lane & 15)) * pitch + (col + ((lane >> 4) << 3)) * 2);
}

// Two floats as the sum of two bf16 pairs.
__device__ __forceinline__ void split2(float a, float b, uint32_t &hi, uint32_t &lo)
{
    hi = ptx::pack_bf16x2(a, b);
    lo = ptx::pack_bf16x2(a - bf16_lo(hi), b - bf16_hi(hi));
}

}  // namespace mma16

__host__ __device__ inline int chunk_smem_bytes(int state)
{
    const int n = (state + 15) / 16 * 16, np = (n + 8) * 2, xp = (kChunkCols + 8) * 2;
    return 2 * kChunk * (2 * np + xp) + 2 * kChunk * xp + 2 * n * xp + 4 * kChunk * 4;
}

__global__ void __launch_bounds__(kChunkThreads)
mamba_chunk_kernel(float *__restrict__ y, const __nv_bfloat16 *__restrict__ xbc, int ld_xbc, const float *__restrict__ dt, const float *__restrict__ log_decay,
                   const float *__restrict__ d_skip, const MambaShape s, const StepEntry *__restrict__ entries)
{
    using namespace mma16;
    extern __shared__ __align__(16) uint8_t chunk_smem[];
    const int slices = (s.vdim + kChunkCols - 1) / kChunkCols;
    const int h = blockIdx.x / slices, p0 = (blockIdx.x % slices) * kChunkCols;
    const int P = s.vdim, N = s.state, n16 = (N + 15) / 16, NP = n16 * 16;
    const int g = h / (s.heads / s.groups);
    const int cols = min(kChunkCols, P - p0);
    const int np = (NP + 8) * 2, xp = (kChunkCols + 8) * 2;   // row pitches in bytes
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // shared memory: two buffers of [B | C | x], scaled x (two terms), state (two terms), per-token values
    const int buf_bytes = kChunk * (2 * np + xp);
    const uint32_t base = ptx::smem_u32(chunk_smem);
    const uint32_t wx = base + 2 * buf_bytes, st = wx + 2 * kChunk * xp;
    float *cum = reinterpret_cast<float *>(chunk_smem + 2 * buf_bytes + 2 * kChunk * xp + 2 * NP * xp), *step = cum + kChunk, *up = step + kChunk, *down = up + kChunk;
    auto tile_b = [&](int b) { return base + b * buf_bytes; };
    auto tile_c = [&](int b) { return base + b * buf_bytes + kChunk * np; };
    auto tile_x = [&](int b) { return base + b * buf_bytes + 2 * kChunk * np; };

    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[blockIdx.y];
    float *state = reinterpret_cast<float *>(e.slot + s.ssm_state) + static_cast<long long>(h) * N * P + p0;
    const bool vec = P % 8 == 0 && N % 8 == 0;    // all column offsets are then multiples of 8
    const int off_b = s.inner + g * N, off_c = off_b + s.groups * N;

    // One piece of eight columns of a row: 16-byte asynchronous copy, or plain loads where columns are unaligned or end.
    auto piece = [&](uint32_t dst, const __nv_bfloat16 *src, int have) {
        if (vec && have >= 8) {
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
        } else {
            uint32_t w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t a = 2 * i < have ? __bfloat16_as_ushort(src[2 * i]) : 0u, b = 2 * i + 1 < have ? __bfloat16_as_ushort(src[2 * i + 1]) : 0u;
                w[i] = a | b << 16;
            }
            ptx::sts128(dst, w[0], w[1], w[2], w[3]);
        }
    };
    auto fetch = [&](int chunk, int b) {
        const int t0 = chunk * kChunk;
        const int per_row = 2 * (NP / 8) + kChunkCols / 8;
        for (int i = threadIdx.x; i < kChunk * per_row; i += kChunkThreads) {
            const int t = i / per_row, q = i % per_row;
            const bool in = t0 + t < e.count;
            const __nv_bfloat16 *row = xbc + static_cast<long long>(e.row0 + (in ? t0 + t : 0)) * ld_xbc;
            if (q < NP / 8)
                piece(tile_b(b) + t * np + q * 16, row + off_b + q * 8, in ? min(8, N - q * 8) : 0);
            else if (q < 2 * (NP / 8))
                piece(tile_c(b) + t * np + (q - NP / 8) * 16, row + off_c + (q - NP / 8) * 8, in ? min(8, N - (q - NP / 8) * 8) : 0);
            else
                piece(tile_x(b) + t * xp + (q - 2 * (NP / 8)) * 16, row + h * P + p0 + (q - 2 * (NP / 8)) * 8, in ? min(8, cols - (q - 2 * (NP / 8)) * 8) : 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    // state fragments: row tile (warp + 4 k) of 16 state rows, four tiles of 8 columns
    float S[2][4][4];
    const int r = lane >> 2, c2 = (lane & 3) * 2;
#pragma unroll
    for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int n = (warp + 4 * k) * 16 + r + (i >> 1) * 8, p = j * 8 + c2 + (i & 1);
                S[k][j][i] = n < N && p < cols ? state[static_cast<long long>(n) * P + p] : 0.0f;
            }
    const float skip = d_skip[h];
    const int chunks = (e.count + kChunk - 1) / kChunk;
    fetch(0, 0);
    for (int ch = 0; ch < chunks; ++ch) {
        const int b = ch & 1, t0 = ch * kChunk;
        if (ch + 1 < chunks) {
            fetch(ch + 1, b ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        if (warp == 0) {   // running sums of the log-decays: two tokens per lane
            float v[2], d[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int t = t0 + 2 * lane + i;
                const long long at = static_cast<long long>(e.row0 + t) * s.heads + h;
                v[i] = t < e.count ? log_decay[at] : 0.0f;
                d[i] = t < e.count ? dt[at] : 0.0f;
            }
            float sum = v[0] + v[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float u = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += u;
            }
            const float end = __shfl_sync(0xffffffffu, sum, 31);
            const float c1 = sum, c0 = sum - v[1];
            cum[2 * lane] = c0;
            cum[2 * lane + 1] = c1;
            step[2 * lane] = d[0];
            step[2 * lane + 1] = d[1];
            up[2 * lane] = expf(c0);
            up[2 * lane + 1] = expf(c1);
            down[2 * lane] = expf(end - c0) * d[0];
            down[2 * lane + 1] = expf(end - c1) * d[1];
        }
        __syncthreads();
        // scaled x and the state before the chunk, as two bf16 terms each
        for (int i = threadIdx.x; i < kChunk * (kChunkCols / 2); i += kChunkThreads) {
            const int t = i / (kChunkCols / 2), q = i % (kChunkCols / 2);
            uint32_t xv, hi, lo;
            asm volatile("ld.shared.b32 %0, [%1];" : "=r"(xv) : "r"(tile_x(b) + t * xp + q * 4) : "memory");
            split2(down[t] * bf16_lo(xv), down[t] * bf16_hi(xv), hi, lo);
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(wx + t * xp + q * 4), "r"(hi) : "memory");
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(wx + kChunk * xp + t * xp + q * 4), "r"(lo) : "memory");
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            if (warp + 4 * k < n16) {
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        uint32_t hi, lo;
                        split2(S[k][j][2 * half], S[k][j][2 * half + 1], hi, lo);
                        const uint32_t at = st + ((warp + 4 * k) * 16 + r + 8 * half) * xp + (j * 8 + c2) * 2;
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(at), "r"(hi) : "memory");
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(at + NP * xp), "r"(lo) : "memory");
                    }
            }
        }
        __syncthreads();
        // this warp's 16 rows of the chunk: contribution of the state, scores against the chunk's keys
        float Y[4][4] = {}, G[8][4] = {};
        for (int k = 0; k < n16; ++k) {
            uint32_t a[4], f[4];
            a_frag(a, tile_c(b), np, warp * 16, k * 16, lane);
#pragma unroll
            for (int term = 0; term < 2; ++term)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    b_frag_t(f, st + term * NP * xp, xp, k * 16, j * 16, lane);
                    mma(Y[2 * j], a, f[0], f[1]);
                    mma(Y[2 * j + 1], a, f[2], f[3]);
                }
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (j <= warp) {
                    b_frag(f, tile_b(b), np, j * 16, k * 16, lane);
                    mma(G[2 * j], a, f[0], f[1]);
                    mma(G[2 * j + 1], a, f[2], f[3]);
                }
        }
        const int ta = warp * 16 + r, tb = ta + 8;
        const float ua = up[ta], ub = up[tb], ca = cum[ta], cb = cum[tb];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            Y[j][0] *= ua;
            Y[j][1] *= ua;
            Y[j][2] *= ub;
            Y[j][3] *= ub;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk > warp) continue;
            // 16 keys as the A operand: decayed, stepped, causal
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                const int key = kk * 16 + q * 8 + c2;
                float (&gq)[4] = G[2 * kk + q];
                const float s0 = step[key], s1 = step[key + 1], k0 = cum[key], k1 = cum[key + 1];
                const float w00 = key <= ta ? gq[0] * expf(ca - k0) * s0 : 0.0f, w01 = key + 1 <= ta ? gq[1] * expf(ca - k1) * s1 : 0.0f;
                const float w10 = key <= tb ? gq[2] * expf(cb - k0) * s0 : 0.0f, w11 = key + 1 <= tb ? gq[3] * expf(cb - k1) * s1 : 0.0f;
                split2(w00, w01, hi[2 * q], lo[2 * q]);
                split2(w10, w11, hi[2 * q + 1], lo[2 * q + 1]);
            }
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                uint32_t f[4];
                b_frag_t(f, tile_x(b), xp, kk * 16, j * 16, lane);
                mma(Y[2 * j], hi, f[0], f[1]);
                mma(Y[2 * j], lo, f[0], f[1]);
                mma(Y[2 * j + 1], hi, f[2], f[3]);
                mma(Y[2 * j + 1], lo, f[2], f[3]);
            }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = half ? tb : ta;
            if (t0 + t < e.count) {
                float *dst = y + static_cast<long long>(e.row0 + t0 + t) * s.inner + h * P + p0;
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int p = j * 8 + c2;
                    uint32_t xv;
                    asm volatile("ld.shared.b32 %0, [%1];" : "=r"(xv) : "r"(tile_x(b) + t * xp + p * 2) : "memory");
                    const float v0 = fmaf(skip, bf16_lo(xv), Y[j][2 * half]), v1 = fmaf(skip, bf16_hi(xv), Y[j][2 * half + 1]);
                    if (vec && p + 1 < cols) {
                        *reinterpret_cast<float2 *>(dst + p) = make_float2(v0, v1);
                    } else {
                        if (p < cols) dst[p] = v0;
                        if (p + 1 < cols) dst[p + 1] = v1;
                    }
                }
            }
        }
        // the state after the chunk
        const float keep = up[kChunk - 1];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            if (warp + 4 * k < n16) {
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int i = 0; i < 4; ++i) S[k][j][i] *= keep;
#pragma unroll
                for (int kk = 0; kk < kChunk / 16; ++kk) {
                    uint32_t a[4], f[4];
                    a_frag_t(a, tile_b(b), np, kk * 16, (warp + 4 * k) * 16, lane);
#pragma unroll
                    for (int term = 0; term < 2; ++term)
#pragma unroll
                        for (int j = 0; j < 2; ++j) {
                            b_frag_t(f, wx + term * kChunk * xp, xp, kk * 16, j * 16, lane);
                            mma(S[k][2 * j], a, f[0], f[1]);
                            mma(S[k][2 * j + 1], a, f[2], f[3]);
                        }
                }
            }
        }
        __syncthreads();   // the buffers may be overwritten
    }
#pragma unroll
    for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int n = (warp + 4 * k) * 16 + r + (i >> 1) * 8, p = j * 8 + c2 + (i & 1);
                if (n < N && p < cols) state[static_cast<long long>(n) * P + p] = S[k][j][i];
            }
}

}  // namespace dec
}  // namespace gptb200
