// The wkv recurrence (linear_attention.cuh) over prompts: chunks of 16 tokens on tensor cores, segments side by side.
//
// With A_t[c] the running sum of a chunk's log-decays of key channel c up to token t and S the state before the chunk,
//   o_t = (r_t exp(A_{t-1})) S + sum_{s < t} (sum_c r_t[c] k_s[c] exp(A_{t-1}[c] - A_s[c])) v_s + (r_t . u k_t) v_t
//   S  <- diag(exp(A_end)) S + sum_s (k_s exp(A_end - A_s)) v_s^T
// No exponent is positive, so nothing can overflow however strong the decays are; this is what limits a chunk to 16 tokens (the scores
// inside it have no common factor per token and are summed up channel by channel in fp32).
//
// A block carries one head through the tokens of a request or of a segment of it.  Every warp keeps S^T for 16 value columns in fp32
// accumulators, which are at the same time the layout of an A operand: the state goes into the next product from registers.  What is
// fp32 by nature (state, decayed r and k, scores) enters a product as the sum of two bf16 values.  The head's norm and the gate are applied
// on the way out.
//
// Segments: a first launch computes what each segment alone adds to the state and how much it lets earlier state decay, a second one
// turns those into the segments' initial states, the third computes the outputs.
#pragma once

#include "attention_prefill_sm100.cuh"   // exp2_approx
#include "linear_attention.cuh"
#include "mamba2_chunk.cuh"   // mma16

namespace gptb200 {
namespace dec {

constexpr int kWkvChunk = 16;
constexpr int kWkvMaxDim = 128;

// blocks per SM that registers and shared memory allow
__host__ __device__ constexpr int wkv_blocks(int kt) { return kt == 8 ? 2 : kt == 4 ? 4 : 8; }

struct WkvChunkLayout {
    int xp, fp;                     // row pitches of bf16 tiles (bytes) and fp32 tiles (floats)
    int tile, raw, buf;             // bytes: bf16 tile, offset of the fp32 tile in a buffer, one buffer
    int cum_before, cum, r_hi, r_lo, k_hi, k_lo, p_hi, p_lo, end, red, total;
};

__host__ __device__ constexpr WkvChunkLayout wkv_chunk_layout(int kt)
{
    WkvChunkLayout l{};
    l.xp = (16 * kt + 8) * 2;
    l.fp = 16 * kt + 4;
    l.tile = kWkvChunk * l.xp;
    l.raw = 4 * l.tile;
    l.buf = l.raw + kWkvChunk * l.fp * 4;
    l.cum_before = 2 * l.buf;
    l.cum = l.cum_before + kWkvChunk * l.fp * 4;
    l.r_hi = l.cum + kWkvChunk * l.fp * 4;
    l.r_lo = l.r_hi + l.tile;
    l.k_hi = l.r_lo + l.tile;
    l.k_lo = l.k_hi + l.tile;
    l.p_hi = l.k_lo + l.tile;
    l.p_lo = l.p_hi + kWkvChunk * 48;
    l.end = l.p_lo + kWkvChunk * 48;
    l.red = l.end + 16 * kt * 4;
    l.total = l.red + kt * kWkvChunk * 4;
    return l;
}

// tanh of W1 x as the sum of two bf16 values: [high: rank_pad | low: rank_pad], the rows that W2 | W2 multiplies.
__global__ void wkv_low_rank_kernel(__nv_bfloat16 *__restrict__ out, int rank_pad, const float *__restrict__ low, int ld_low, int rank)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const long long row = blockIdx.x;
    for (int i = threadIdx.x; i < rank_pad; i += blockDim.x) {
        const float v = i < rank ? tanhf(low[row * ld_low + i]) : 0.0f;
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        out[row * 2 * rank_pad + i] = hi;
        out[row * 2 * rank_pad + rank_pad + i] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
}

// KT: tiles of 16 channels (heads of up to 16 * KT), one warp each.  raw [rows][ld_raw]: W2 tanh(W1 x).  segment_state
// [entry][head][segment][dim][dim], segment_decay [entry][head][segment][dim].  grid: (heads, entries, segments)
template <int KT, bool SEGMENT_STATES>
__global__ void __launch_bounds__(32 * KT, wkv_blocks(KT))
wkv_chunk_kernel(__nv_bfloat16 *__restrict__ out, int ld_out, const __nv_bfloat16 *__restrict__ proj, const float *__restrict__ raw, int ld_raw, const float *__restrict__ w0,
                 const float *__restrict__ bonus, const float *__restrict__ weight, float eps, const WkvShape s, const StepEntry *__restrict__ entries, int segment_tokens, int max_segments,
                 float *__restrict__ segment_state, float *__restrict__ segment_decay)
{
    using namespace mma16;
    constexpr WkvChunkLayout L = wkv_chunk_layout(KT);
    constexpr int DP = 16 * KT, THREADS = 32 * KT;
    constexpr float kLog2e = 1.4426950408889634f;
    extern __shared__ __align__(16) uint8_t wkv_smem[];
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[blockIdx.y];
    const int segment = blockIdx.z, begin = segment * segment_tokens;
    const bool last_segment = begin + segment_tokens >= e.count;
    if (begin >= e.count || (SEGMENT_STATES && last_segment)) return;
    const int count = min(segment_tokens, e.count - begin);
    const long long first_row = e.row0 + begin;
    const int h = blockIdx.x, D = s.dim, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t base = ptx::smem_u32(wkv_smem);
    auto floats = [&](int at) { return reinterpret_cast<float *>(wkv_smem + at); };
    auto halves = [&](int at) { return reinterpret_cast<__nv_bfloat16 *>(wkv_smem + at); };
    const bool vec = D % 8 == 0 && ld_raw % 4 == 0;   // the groups' columns and pitches are multiples of 8

    // one chunk's r, k, v, gate and raw decays; rows beyond the segment and channels beyond the head are zero
    auto fetch = [&](int chunk, int b) {
        const int at = b * L.buf;
        for (int i = tid; i < kWkvChunk * (DP / 8) * 4; i += THREADS) {
            const int c = i % (DP / 8) * 8, t = i / (DP / 8) % kWkvChunk, g = i / (DP / 8) / kWkvChunk;
            if (SEGMENT_STATES && (g == 0 || g == 3)) continue;
            const int have = chunk * kWkvChunk + t < count ? min(8, D - c) : 0;
            const __nv_bfloat16 *src = proj + (first_row + chunk * kWkvChunk + t) * s.ld + g * s.group + h * D + c;
            const uint32_t dst = base + at + g * L.tile + t * L.xp + c * 2;
            if (vec && have == 8) {
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
            } else {
                uint32_t w[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const uint32_t lo = 2 * j < have ? __bfloat16_as_ushort(src[2 * j]) : 0u, hi = 2 * j + 1 < have ? __bfloat16_as_ushort(src[2 * j + 1]) : 0u;
                    w[j] = lo | hi << 16;
                }
                ptx::sts128(dst, w[0], w[1], w[2], w[3]);
            }
        }
        for (int i = tid; i < kWkvChunk * (DP / 4); i += THREADS) {
            const int c = i % (DP / 4) * 4, t = i / (DP / 4);
            const int have = chunk * kWkvChunk + t < count ? min(4, D - c) : 0;
            const float *src = raw + (first_row + chunk * kWkvChunk + t) * ld_raw + h * D + c;
            const uint32_t dst = base + at + L.raw + (t * L.fp + c) * 4;
            if (vec && have == 4) {
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
            } else {
                float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (have > 0) v.x = src[0];
                if (have > 1) v.y = src[1];
                if (have > 2) v.z = src[2];
                if (have > 3) v.w = src[3];
                store4(floats(at + L.raw) + t * L.fp + c, v);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    const int r = lane >> 2, c2 = (lane & 3) * 2;
    const int col = warp * 16 + r;                      // this thread's value columns: col, col + 8
    const long long seg0 = (static_cast<long long>(blockIdx.y) * s.heads + h) * max_segments;
    float *state = reinterpret_cast<float *>(e.slot + s.state) + static_cast<long long>(h) * D * D;
    const long long copy = static_cast<long long>(s.heads) * D * D;
    // S^T: rows = value columns, columns = key channels
    float S[2 * KT][4];
    auto each = [&](auto &&f) {
#pragma unroll
        for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int n = j * 8 + c2 + (i & 1), p = col + (i >> 1) * 8;
                f(S[j][i], n < D && p < D, n * D + p);
            }
    };
    fetch(0, 0);
    if (SEGMENT_STATES) {
        each([&](float &v, bool, int) { v = 0.0f; });
    } else {
        const float *init = segment == 0 ? state + e.parity * copy : segment_state + (seg0 + segment - 1) * D * D;
        each([&](float &v, bool ok, int at) { v = ok ? init[at] : 0.0f; });
    }
    const int ch = tid >> 1, half = tid & 1;            // step 1: two threads per channel, eight tokens each
    const float channel_w0 = ch < D ? w0[h * D + ch] : 0.0f;
    float decay_sum = 0.0f;
    if (!SEGMENT_STATES)
        for (int i = tid; i < 2 * kWkvChunk * 24; i += THREADS) halves(L.p_hi)[i] = __float2bfloat16_rn(0.0f);   // scores beyond the diagonal stay zero
    const float weight_a = !SEGMENT_STATES && col < D ? weight[h * D + col] : 0.0f, weight_b = !SEGMENT_STATES && col + 8 < D ? weight[h * D + col + 8] : 0.0f;
    const int chunks = (count + kWkvChunk - 1) / kWkvChunk;
    for (int chunk = 0; chunk < chunks; ++chunk) {
        const int b = chunk & 1, at = b * L.buf;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // this chunk's tiles are there; everything of the chunk before has been read
        if (chunk + 1 < chunks) fetch(chunk + 1, b ^ 1);
        // 1. running log2-decays, decayed r and k
        {
            float sum[8], run = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int t = half * 8 + i;
                // beyond 2^-160 nothing is left of a value in fp32
                if (chunk * kWkvChunk + t < count) run -= fminf(expf(floats(at + L.raw)[t * L.fp + ch] + channel_w0) * kLog2e, 160.0f);
                sum[i] = run;
            }
            const float other = __shfl_xor_sync(0xffffffffu, run, 1), start = half ? other : 0.0f, all = run + other;
            decay_sum += all;
            if (half == 0) floats(L.end)[ch] = ptx_attn::exp2_approx(all);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int t = half * 8 + i;
                const float before = start + (i ? sum[i - 1] : 0.0f), now = start + sum[i];
                const float kd = __bfloat162float(halves(at + L.tile + t * L.xp)[ch]) * ptx_attn::exp2_approx(all - now);
                const __nv_bfloat16 kh = __float2bfloat16_rn(kd);
                halves(L.k_hi + t * L.xp)[ch] = kh;
                halves(L.k_lo + t * L.xp)[ch] = __float2bfloat16_rn(kd - __bfloat162float(kh));
                if (!SEGMENT_STATES) {
                    floats(L.cum_before)[t * L.fp + ch] = before;
                    floats(L.cum)[t * L.fp + ch] = now;
                    const float rd = __bfloat162float(halves(at + t * L.xp)[ch]) * ptx_attn::exp2_approx(before);
                    const __nv_bfloat16 rh = __float2bfloat16_rn(rd);
                    halves(L.r_hi + t * L.xp)[ch] = rh;
                    halves(L.r_lo + t * L.xp)[ch] = __float2bfloat16_rn(rd - __bfloat162float(rh));
                }
            }
        }
        __syncthreads();
        if (!SEGMENT_STATES) {
            // 2. scores inside the chunk: 36 blocks of 2 x 2 on and below the diagonal, four threads (a quarter of the channels) each
#pragma unroll 1
            for (int item = tid; item < (144 + 31) / 32 * 32; item += THREADS) {
                const int quarter = item & 3, blk = min(item >> 2, 35);
                int bi = 0, bj = blk;
                while (bj > bi) bj -= ++bi;
                const bool diagonal = bi == bj;
                float acc[2][2] = {};
#pragma unroll 1
                for (int c = 4 * quarter; c < DP; c += 16) {
                    float4 rv[2], kv[2], rb[2], kc[2];
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        rv[i] = load4(halves(at + (2 * bi + i) * L.xp) + c);
                        kv[i] = load4(halves(at + L.tile + (2 * bj + i) * L.xp) + c);
                        rb[i] = load4(floats(L.cum_before) + (2 * bi + i) * L.fp + c);
                        kc[i] = load4(floats(L.cum) + (2 * bj + i) * L.fp + c);
                    }
                    float4 u = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    if (diagonal) {
                        const float *src = bonus + h * D + c;
                        if (c + 4 <= D) {
                            u = make_float4(__ldg(src), __ldg(src + 1), __ldg(src + 2), __ldg(src + 3));
                        } else {
                            if (c < D) u.x = __ldg(src);
                            if (c + 1 < D) u.y = __ldg(src + 1);
                            if (c + 2 < D) u.z = __ldg(src + 2);
                        }
                    }
#pragma unroll
                    for (int i = 0; i < 2; ++i)
#pragma unroll
                        for (int j = 0; j < 2; ++j) {
                            const bool own = diagonal && i == j;
                            auto term = [&](float x, float y, float before, float now, float uc) {
                                acc[i][j] = fmaf(x * y, own ? uc : ptx_attn::exp2_approx(before - now), acc[i][j]);
                            };
                            if (diagonal && j > i) continue;   // a later key
                            term(rv[i].x, kv[j].x, rb[i].x, kc[j].x, u.x);
                            term(rv[i].y, kv[j].y, rb[i].y, kc[j].y, u.y);
                            term(rv[i].z, kv[j].z, rb[i].z, kc[j].z, u.z);
                            term(rv[i].w, kv[j].w, rb[i].w, kc[j].w, u.w);
                        }
                }
#pragma unroll
                for (int i = 0; i < 2; ++i) {
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        acc[i][j] += __shfl_xor_sync(0xffffffffu, acc[i][j], 1);
                        acc[i][j] += __shfl_xor_sync(0xffffffffu, acc[i][j], 2);
                    }
                    if (quarter == i && item < 144) {
                        uint32_t hi, lo;
                        split2(acc[i][0], acc[i][1], hi, lo);
                        *reinterpret_cast<uint32_t *>(wkv_smem + L.p_hi + (2 * bi + i) * 48 + 4 * bj) = hi;
                        *reinterpret_cast<uint32_t *>(wkv_smem + L.p_lo + (2 * bi + i) * 48 + 4 * bj) = lo;
                    }
                }
            }
            __syncthreads();
        }
        // 3. this warp's 16 value columns
        uint32_t va[4];
        a_frag_t(va, base + at + 2 * L.tile, L.xp, 0, warp * 16, lane);
        if (!SEGMENT_STATES) {
            float O[2][4] = {};
            uint32_t f[4];
            b_frag(f, base + L.p_hi, 48, 0, 0, lane);
            mma(O[0], va, f[0], f[1]);
            mma(O[1], va, f[2], f[3]);
            b_frag(f, base + L.p_lo, 48, 0, 0, lane);
            mma(O[0], va, f[0], f[1]);
            mma(O[1], va, f[2], f[3]);
#pragma unroll
            for (int kt = 0; kt < KT; ++kt) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int q = 0; q < 4; ++q) split2(S[2 * kt + (q >> 1)][2 * (q & 1)], S[2 * kt + (q >> 1)][2 * (q & 1) + 1], hi[q], lo[q]);
                b_frag(f, base + L.r_hi, L.xp, 0, kt * 16, lane);
                mma(O[0], hi, f[0], f[1]);
                mma(O[1], hi, f[2], f[3]);
                mma(O[0], lo, f[0], f[1]);
                mma(O[1], lo, f[2], f[3]);
                b_frag(f, base + L.r_lo, L.xp, 0, kt * 16, lane);
                mma(O[0], hi, f[0], f[1]);
                mma(O[1], hi, f[2], f[3]);
            }
            // the head's norm: sums over the value columns of each token
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    float ss = O[j][i] * O[j][i] + O[j][i + 2] * O[j][i + 2];
                    ss += __shfl_xor_sync(0xffffffffu, ss, 4);
                    ss += __shfl_xor_sync(0xffffffffu, ss, 8);
                    ss += __shfl_xor_sync(0xffffffffu, ss, 16);
                    if (r == 0) floats(L.red)[warp * kWkvChunk + j * 8 + c2 + i] = ss;
                }
            __syncthreads();   // also: the decayed r have been read, their place takes the outputs
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int t = j * 8 + c2 + i;
                    float ss = 0.0f;
#pragma unroll
                    for (int w = 0; w < KT; ++w) ss += floats(L.red)[w * kWkvChunk + t];
                    const float inv = rsqrtf(ss / D + eps);
                    const __nv_bfloat16 *gate = halves(at + 3 * L.tile + t * L.xp);
                    __nv_bfloat16 *dst = halves(L.r_hi + t * L.xp);
                    dst[col] = __float2bfloat16_rn(O[j][i] * inv * weight_a * silu_t<__nv_bfloat16>(__bfloat162float(gate[col])));
                    dst[col + 8] = __float2bfloat16_rn(O[j][i + 2] * inv * weight_b * silu_t<__nv_bfloat16>(__bfloat162float(gate[col + 8])));
                }
        }
        // the state after the chunk
        {
            const float *end = floats(L.end);
#pragma unroll
            for (int kt = 0; kt < KT; ++kt) {
#pragma unroll
                for (int j = 2 * kt; j < 2 * kt + 2; ++j) {
                    const float2 d = *reinterpret_cast<const float2 *>(end + j * 8 + c2);
                    S[j][0] *= d.x;
                    S[j][1] *= d.y;
                    S[j][2] *= d.x;
                    S[j][3] *= d.y;
                }
                uint32_t f[4];
                b_frag_t(f, base + L.k_hi, L.xp, 0, kt * 16, lane);
                mma(S[2 * kt], va, f[0], f[1]);
                mma(S[2 * kt + 1], va, f[2], f[3]);
                b_frag_t(f, base + L.k_lo, L.xp, 0, kt * 16, lane);
                mma(S[2 * kt], va, f[0], f[1]);
                mma(S[2 * kt + 1], va, f[2], f[3]);
            }
        }
        if (!SEGMENT_STATES) {
            __syncthreads();
            for (int i = tid; i < kWkvChunk * (DP / 8); i += THREADS) {
                const int c = i % (DP / 8) * 8, t = i / (DP / 8);
                if (chunk * kWkvChunk + t >= count || c >= D) continue;
                const __nv_bfloat16 *src = halves(L.r_hi + t * L.xp) + c;
                __nv_bfloat16 *dst = out + (first_row + chunk * kWkvChunk + t) * ld_out + h * D + c;
                if (vec)
                    *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(src);
                else
                    for (int j = 0; j < min(8, D - c); ++j) dst[j] = src[j];
            }
        }
    }
    if (SEGMENT_STATES || last_segment) {
        float *dst = SEGMENT_STATES ? segment_state + (seg0 + segment) * D * D : state + (e.parity ^ 1) * copy;
        each([&](float &v, bool ok, int i) {
            if (ok) dst[i] = v;
        });
        if (SEGMENT_STATES && half == 0 && ch < D) segment_decay[(seg0 + segment) * D + ch] = ptx_attn::exp2_approx(decay_sum);
    }
}

// What the segments add -> the states after them: segment_state[i] <- decay_i * (state before) + segment_state[i].
// grid: (heads * blocks of 256 state values, entries)
__global__ void wkv_segments_kernel(float *__restrict__ segment_state, const float *__restrict__ segment_decay, const WkvShape s, const StepEntry *__restrict__ entries, int segment_tokens,
                                    int max_segments)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const int D = s.dim, blocks = (D * D + 255) / 256, h = blockIdx.x / blocks, at = blockIdx.x % blocks * 256 + threadIdx.x;
    if (at >= D * D) return;
    const StepEntry e = entries[blockIdx.y];
    const float *state = reinterpret_cast<const float *>(e.slot + s.state) + (static_cast<long long>(e.parity) * s.heads + h) * D * D;
    const long long seg0 = (static_cast<long long>(blockIdx.y) * s.heads + h) * max_segments;
    const int segments = (e.count + segment_tokens - 1) / segment_tokens;
    float v = state[at];
    for (int i = 0; i + 1 < segments; ++i) {
        float *add = segment_state + (seg0 + i) * D * D + at;
        v = fmaf(v, segment_decay[(seg0 + i) * D + at / D], *add);
        *add = v;
    }
}

}  // namespace dec
}  // namespace gptb200
