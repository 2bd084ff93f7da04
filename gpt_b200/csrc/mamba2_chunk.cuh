// Recurrences with one decay per head and token (Mamba-2; linear attention with constant decays: steps of one, no skip) over prompts: the
// state-space duality form in chunks of 64 tokens, on tensor cores.
//
// With a_t the running sum of log-decays inside a chunk and S the state before it,
//   y_t = exp(a_t) C_t S + sum_{s <= t} exp(a_t - a_s) dt_s (C_t . B_s) x_s + D x_t
//   S  <- exp(a_end) S + sum_s exp(a_end - a_s) dt_s B_s x_s^T
// One block carries one head's state for 32 of its value columns through the chunks of a request, or of a segment of it: S stays in
// fp32 accumulators from chunk to chunk, and the next chunk's x, B and C arrive while this one is computed.  Four warps
// compute the outputs, four the state.  x, B and C are bf16 as the convolution left them; everything that is fp32 by nature (weights with
// decays and steps, the scaled x, the state) enters a product as the sum of two bf16 values.
//
// Long requests are cut into segments that run side by side: a first launch computes what each segment alone adds to the state and by
// how much it lets earlier state decay; in the second every block puts its segment's initial state together from those.
#pragma once

#include "mamba2.cuh"

namespace gptb200 {
namespace dec {

constexpr int kChunk = 64;
constexpr int kChunkCols = 32;       // value columns per block
constexpr int kChunkThreads = 256;
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
    return 2 * kChunk * (2 * np + xp) + 2 * kChunk * xp + 2 * n * xp + 2 * 4 * kChunk * 4;
}

// SEGMENT_STATES: only what a segment adds to the state, from zero, into segment_state [entry][head][segment][state][vdim] and the
// segment's decay into segment_decay [entry][head][segment]; the last segment is left out.  Otherwise outputs and, in the last
// segment, the request's new state.  dt null: steps of one; ld_decay: row pitch of log_decay (0: constant decays); d_skip null: none.
// grid: (heads * column slices, entries, segments)
template <bool SEGMENT_STATES>
__global__ void __launch_bounds__(kChunkThreads, 2)
mamba_chunk_kernel(float *__restrict__ y, const __nv_bfloat16 *__restrict__ xbc, int ld_xbc, const float *__restrict__ dt, const float *__restrict__ log_decay, int ld_decay,
                   const float *__restrict__ d_skip, const RecurrentShape s, const StepEntry *__restrict__ entries, int segment_tokens, int max_segments, float *__restrict__ segment_state,
                   float *__restrict__ segment_decay)
{
    using namespace mma16;
    extern __shared__ __align__(16) uint8_t chunk_smem[];
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[blockIdx.y];
    const int segment = blockIdx.z, begin = segment * segment_tokens;
    const bool last_segment = begin + segment_tokens >= e.count;
    if (begin >= e.count || (SEGMENT_STATES && last_segment)) return;
    const int count = min(segment_tokens, e.count - begin), first_row = e.row0 + begin;

    const int slices = (s.vdim + kChunkCols - 1) / kChunkCols;
    const int h = blockIdx.x / slices, p0 = (blockIdx.x % slices) * kChunkCols;
    const int P = s.vdim, N = s.state, n16 = (N + 15) / 16, NP = n16 * 16;
    const int g = h / (s.heads / s.groups);
    const int cols = min(kChunkCols, P - p0);
    const int np = (NP + 8) * 2, xp = (kChunkCols + 8) * 2;   // row pitches in bytes
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool state_role = warp >= 4;
    const int rw = warp & 3;      // warp within its role
    // shared memory: two buffers of [B | C | x], scaled x (two terms), state (two terms), per-token values of two chunks
    const int buf_bytes = kChunk * (2 * np + xp);
    const uint32_t base = ptx::smem_u32(chunk_smem);
    const uint32_t wx = base + 2 * buf_bytes, st = wx + 2 * kChunk * xp;
    float *tokens = reinterpret_cast<float *>(chunk_smem + 2 * buf_bytes + 2 * kChunk * xp + 2 * NP * xp);
    auto tile_b = [&](int b) { return base + b * buf_bytes; };
    auto tile_c = [&](int b) { return base + b * buf_bytes + kChunk * np; };
    auto tile_x = [&](int b) { return base + b * buf_bytes + 2 * kChunk * np; };
    // running log2-decay, step, decay since the chunk's start, decay to its end times step
    auto cum = [&](int b) { return tokens + b * 4 * kChunk; };
    auto step = [&](int b) { return tokens + b * 4 * kChunk + kChunk; };
    auto up = [&](int b) { return tokens + b * 4 * kChunk + 2 * kChunk; };
    auto down = [&](int b) { return tokens + b * 4 * kChunk + 3 * kChunk; };

    const long long state_floats = static_cast<long long>(s.heads) * N * P;
    float *state = reinterpret_cast<float *>(e.slot + s.ssm_state) + static_cast<long long>(h) * N * P + p0;
    const float *old_state = state + e.parity * state_floats;
    const long long seg0 = (static_cast<long long>(blockIdx.y) * s.heads + h) * max_segments;
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
    // four threads per token
    auto fetch = [&](int chunk, int b) {
        const int t = threadIdx.x >> 2, q0 = threadIdx.x & 3;
        const bool in = chunk * kChunk + t < count;
        const __nv_bfloat16 *row = xbc + static_cast<long long>(first_row + (in ? chunk * kChunk + t : 0)) * ld_xbc;
        for (int q = q0; q < NP / 8; q += 4) {
            piece(tile_b(b) + t * np + q * 16, row + off_b + q * 8, in ? min(8, N - q * 8) : 0);
            if (!SEGMENT_STATES) piece(tile_c(b) + t * np + q * 16, row + off_c + q * 8, in ? min(8, N - q * 8) : 0);
        }
        piece(tile_x(b) + t * xp + q0 * 16, row + h * P + p0 + q0 * 8, in ? min(8, cols - q0 * 8) : 0);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // per-token values of a chunk by one warp, two tokens per lane: load early, finish later
    constexpr float kLog2e = 1.4426950408889634f;
    float ld[2], sd[2];
    auto load_tokens = [&](int chunk) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int t = chunk * kChunk + 2 * lane + i;
            const long long row = first_row + t;
            ld[i] = t < count ? log_decay[row * ld_decay + h] * kLog2e : 0.0f;
            sd[i] = t >= count ? 0.0f : dt ? dt[row * s.heads + h] : 1.0f;
        }
    };
    auto finish_tokens = [&](int b) {
        float sum = ld[0] + ld[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += u;
        }
        const float end = __shfl_sync(0xffffffffu, sum, 31), c1 = sum, c0 = sum - ld[1];
        *reinterpret_cast<float2 *>(cum(b) + 2 * lane) = make_float2(c0, c1);
        *reinterpret_cast<float2 *>(step(b) + 2 * lane) = make_float2(sd[0], sd[1]);
        *reinterpret_cast<float2 *>(up(b) + 2 * lane) = make_float2(exp2f(c0), exp2f(c1));
        *reinterpret_cast<float2 *>(down(b) + 2 * lane) = make_float2(exp2f(end - c0) * sd[0], exp2f(end - c1) * sd[1]);
    };

    const int r = lane >> 2, c2 = (lane & 3) * 2;
    // state fragments of the state warps: row tiles rw and rw + 4 of 16 state rows, four tiles of 8 columns
    float S[2][4][4];
    float decay_all = 1.0f;
    fetch(0, 0);
    if (warp == 7) load_tokens(0);
    if (state_role) {
        auto each = [&](auto &&f) {
#pragma unroll
            for (int k = 0; k < 2; ++k)
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int n = (rw + 4 * k) * 16 + r + (i >> 1) * 8, p = j * 8 + c2 + (i & 1);
                        f(S[k][j][i], n < N && p < cols, static_cast<long long>(n) * P + p);
                    }
        };
        if (SEGMENT_STATES) {
            each([&](float &v, bool, long long) { v = 0.0f; });
        } else {
            each([&](float &v, bool ok, long long at) { v = ok ? old_state[at] : 0.0f; });
            for (int i = 0; i < segment; ++i) {
                const float keep = segment_decay[seg0 + i];
                const float *add = segment_state + (seg0 + i) * N * P + p0;
                each([&](float &v, bool ok, long long at) { v = ok ? fmaf(v, keep, add[at]) : 0.0f; });
            }
        }
    }
    if (warp == 7) finish_tokens(0);
    const float skip = d_skip ? d_skip[h] : 0.0f;
    const int chunks = (count + kChunk - 1) / kChunk;
    for (int ch = 0; ch < chunks; ++ch) {
        const int b = ch & 1, t0 = ch * kChunk;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // this chunk's tiles and token values are there, the other buffer is free
        if (ch + 1 < chunks) {
            fetch(ch + 1, b ^ 1);
            if (warp == 7) load_tokens(ch + 1);
        }
        // scaled x and the state before the chunk, as two bf16 terms each
        {
            const float *dn = down(b);
            for (int i = threadIdx.x; i < kChunk * (kChunkCols / 2); i += kChunkThreads) {
                const int t = i / (kChunkCols / 2), q = i % (kChunkCols / 2);
                uint32_t xv, hi, lo;
                asm volatile("ld.shared.b32 %0, [%1];" : "=r"(xv) : "r"(tile_x(b) + t * xp + q * 4) : "memory");
                split2(dn[t] * bf16_lo(xv), dn[t] * bf16_hi(xv), hi, lo);
                asm volatile("st.shared.b32 [%0], %1;" ::"r"(wx + t * xp + q * 4), "r"(hi) : "memory");
                asm volatile("st.shared.b32 [%0], %1;" ::"r"(wx + kChunk * xp + t * xp + q * 4), "r"(lo) : "memory");
            }
        }
        if (state_role && !SEGMENT_STATES) {
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                if (rw + 4 * k < n16) {
#pragma unroll
                    for (int j = 0; j < 4; ++j)
#pragma unroll
                        for (int half = 0; half < 2; ++half) {
                            uint32_t hi, lo;
                            split2(S[k][j][2 * half], S[k][j][2 * half + 1], hi, lo);
                            const uint32_t at = st + ((rw + 4 * k) * 16 + r + 8 * half) * xp + (j * 8 + c2) * 2;
                            asm volatile("st.shared.b32 [%0], %1;" ::"r"(at), "r"(hi) : "memory");
                            asm volatile("st.shared.b32 [%0], %1;" ::"r"(at + NP * xp), "r"(lo) : "memory");
                        }
                }
            }
        }
        __syncthreads();
        if (state_role) {
            // the state after the chunk
            const float keep = up(b)[kChunk - 1];
            decay_all *= keep;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                if (rw + 4 * k < n16) {
#pragma unroll
                    for (int j = 0; j < 4; ++j)
#pragma unroll
                        for (int i = 0; i < 4; ++i) S[k][j][i] *= keep;
#pragma unroll
                    for (int kk = 0; kk < kChunk / 16; ++kk) {
                        uint32_t a[4], f[4];
                        a_frag_t(a, tile_b(b), np, kk * 16, (rw + 4 * k) * 16, lane);
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
            if (warp == 7 && ch + 1 < chunks) finish_tokens(b ^ 1);
            continue;
        }
        if (SEGMENT_STATES) continue;
        // this warp's 16 rows of the chunk: contribution of the state, scores against the chunk's keys
        float Y[4][4] = {}, G[8][4] = {};
        for (int k = 0; k < n16; ++k) {
            uint32_t a[4], f[4];
            a_frag(a, tile_c(b), np, rw * 16, k * 16, lane);
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
                if (j <= rw) {
                    b_frag(f, tile_b(b), np, j * 16, k * 16, lane);
                    mma(G[2 * j], a, f[0], f[1]);
                    mma(G[2 * j + 1], a, f[2], f[3]);
                }
        }
        const int ta = rw * 16 + r, tb = ta + 8;
        const float ua = up(b)[ta], ub = up(b)[tb], ca = cum(b)[ta], cb = cum(b)[tb];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            Y[j][0] *= ua;
            Y[j][1] *= ua;
            Y[j][2] *= ub;
            Y[j][3] *= ub;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk > rw) continue;
            // 16 keys as the A operand: decayed, stepped, causal
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                const int key = kk * 16 + q * 8 + c2;
                float (&gq)[4] = G[2 * kk + q];
                const float2 sk = *reinterpret_cast<const float2 *>(step(b) + key), ck = *reinterpret_cast<const float2 *>(cum(b) + key);
                const float w00 = key <= ta ? gq[0] * exp2f(ca - ck.x) * sk.x : 0.0f, w01 = key + 1 <= ta ? gq[1] * exp2f(ca - ck.y) * sk.y : 0.0f;
                const float w10 = key <= tb ? gq[2] * exp2f(cb - ck.x) * sk.x : 0.0f, w11 = key + 1 <= tb ? gq[3] * exp2f(cb - ck.y) * sk.y : 0.0f;
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
            if (t0 + t < count) {
                float *dst = y + static_cast<long long>(first_row + t0 + t) * s.inner + h * P + p0;
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
    }
    if (state_role && (SEGMENT_STATES || last_segment)) {
        float *dst = SEGMENT_STATES ? segment_state + (seg0 + segment) * N * P + p0 : state + (e.parity ^ 1) * state_floats;
#pragma unroll
        for (int k = 0; k < 2; ++k)
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int n = (rw + 4 * k) * 16 + r + (i >> 1) * 8, p = j * 8 + c2 + (i & 1);
                    if (n < N && p < cols) dst[static_cast<long long>(n) * P + p] = S[k][j][i];
                }
        if (SEGMENT_STATES && p0 == 0 && warp == 4 && lane == 0) segment_decay[seg0 + segment] = decay_all;
    }
}

}  // namespace dec
}  // namespace gptb200
