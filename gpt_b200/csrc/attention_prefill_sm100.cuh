// Causal attention over key and value matrices on the tensor cores (prompts and portions of prompts of one request): latent attention over
// expanded keys and values, grouped attention over its cache.
//
// One CTA takes one head and 256 query rows as two tiles of 128; per block of 128 keys
//   S = Q K^T       tcgen05.mma, Q and K from shared memory (unrotated and rotated parts as separate 64-column blocks), S in TMEM
//   softmax         one thread per row: running maximum and sum in fp32; the weights go back to TMEM over S, each as the sum of two bf16
//                   values (16 bits of mantissa), so that the second product carries more than bf16 weights
//   O += P V        tcgen05.mma with P from TMEM and V from shared memory as stored (MN-major), O in TMEM
// The tiles' chains alternate on the tensor pipe: while one tile's rows are in softmax the other's products run.  O is rescaled
// only when a row's maximum has grown by more than 2^8 since the last time (the sum uses the same reference, so nothing else
// depends on it).  At the end O / sum times the sigmoid gate is stored as bf16.
//
//   warp 0       TMA producer (lane 0): Q once, then K and V blocks through two rings
//   warp 1       MMA issuer (one thread)
//   warps 4-7    softmax and output of tile 0;  warps 8-11: tile 1
// Every wait is bounded, as in the GEMM kernels.
#pragma once

#include "decoder_rows.cuh"

namespace gptb200 {
namespace dec {

struct PrefillParams {
    int rows, pos0;            // the request's rows of this step and the position of the first
    int heads, vdim, v_pad;    // v_pad: value columns per head, a multiple of 16, at most 128
    int kv_share;              // query heads per key / value head
    int q_stride, q_rot;       // words-aligned columns: per head, start of the part whose keys all heads share
    int dim_pad, rot_pad;      // multiples of 16; rot_pad: width of that part (0: none)
    int u_blocks, r_blocks, v_blocks;   // 64-column blocks of the three parts
    int k_stages, v_stages;
    int v_col0;                // first value column of head 0 in the rows of keys and values
    int rot_col0;              // shared key part in its rows
    float scale_log2;          // scale * log2(e)
    float cap_log2, cap_arg;   // CAPPED: cap * log2(e), scale / cap
    __nv_bfloat16 *out;        // [rows][ld_out], head h at h * vdim
    int ld_out;
    const __nv_bfloat16 *gate; // [rows][ld_gate], head h at h * vdim
    long long ld_gate;
    int *status;
};

constexpr int kPrefillThreads = 384;
constexpr int kPrefillBlock = 128 * 128;   // bytes of one [128 rows x 64 bf16] block
constexpr int kPrefillMaxStages = 3;

__host__ __device__ inline int prefill_smem_bytes(int u_blocks, int r_blocks, int v_blocks, int k_stages, int v_stages)
{
    return (2 * (u_blocks + r_blocks) + k_stages * (u_blocks + r_blocks) + v_stages * v_blocks) * kPrefillBlock + 1024 + 256;
}

namespace ptx_attn {

// D[tmem] (+)= A[tmem] * B[smem desc], bf16 operands.
__device__ __forceinline__ void mma_f16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t accumulate)
{
    asm volatile(
        "{\n\t.reg .pred P;\n\t"
        "setp.ne.b32 P, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, P;\n\t}"
        :
        : "r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
        : "memory");
}

// registers -> TMEM: thread i of the warp writes lane i, 32 consecutive columns
__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t (&v)[32])
{
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
        :
        : "r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]),
          "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]), "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]), "r"(v[24]), "r"(v[25]),
          "r"(v[26]), "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
        : "memory");
}

__device__ __forceinline__ void tmem_st_32x16(uint32_t taddr, const uint32_t (&v)[16])
{
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        :
        : "r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]),
          "r"(v[13]), "r"(v[14]), "r"(v[15])
        : "memory");
}

__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

__device__ __forceinline__ float exp2_approx(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// two floats in one register pair
__device__ __forceinline__ uint64_t pack2(float a, float b)
{
    uint64_t v;
    asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(a), "f"(b));
    return v;
}
__device__ __forceinline__ void unpack2(uint64_t v, float &a, float &b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b)
{
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c)
{
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}

__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b)
{
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// tanh of two values within [-1, 1]: x times a polynomial in x^2, the Chebyshev fit of degree 7 of tanh(x) / x (largest error 5e-9,
// with fp32 rounding 7e-8).
__device__ __forceinline__ uint64_t tanh_inner2(uint64_t x)
{
    constexpr float c[8] = {1.0f, -0.33333307504653931f, 0.13332527875900269f, -0.053887963294982910f, 0.021501919254660606f, -0.0079579148441553116f, 0.0023032133467495441f,
                            -0.00035729847149923444f};
    const uint64_t u = mul2(x, x);
    uint64_t p = pack2(c[7], c[7]);
#pragma unroll
    for (int i = 6; i >= 0; --i) p = fma2(p, u, pack2(c[i], c[i]));
    return mul2(p, x);
}

__device__ __forceinline__ float rcp_approx(float x)
{
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// cap * tanh(x): cap - 2 cap / (1 + exp(2 x))
__device__ __forceinline__ float capped(float x, float cap) { return fmaf(-2.0f * cap, rcp_approx(1.0f + exp2_approx(x * 2.8853900817779268f)), cap); }

}  // namespace ptx_attn

// grid: (heads, blocks of 256 rows).  map_kv: rows of [keys of all heads | values of all heads]; map_shared: rows with the key part that all heads share.
// CAPPED: scores become cap * tanh(score / cap).  Special-function instructions (exponential, reciprocal) are what this kernel runs out of
// first, so where all scores of a warp's rows lie within the cap tanh is a polynomial; else 1 - 2 / (1 + exp(2 score / cap)).
template <bool CAPPED>
__global__ void __launch_bounds__(kPrefillThreads, 1)
attention_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_shared, const PrefillParams p)
{
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (ptx::smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t *gen = smem_raw + (base - ptx::smem_u32(smem_raw));
    const int qk_blocks = p.u_blocks + p.r_blocks;
    const uint32_t q_base = base;
    const uint32_t k_base = q_base + 2 * qk_blocks * kPrefillBlock;
    const uint32_t v_base = k_base + p.k_stages * qk_blocks * kPrefillBlock;
    const uint32_t bar = v_base + p.v_stages * p.v_blocks * kPrefillBlock;
    auto q_full = [&](int g) { return bar + 8u * g; };
    auto k_full = [&](int s) { return bar + 8u * (2 + s); };
    auto k_empty = [&](int s) { return bar + 8u * (5 + s); };
    auto v_full = [&](int s) { return bar + 8u * (8 + s); };
    auto v_empty = [&](int s) { return bar + 8u * (11 + s); };
    auto s_full = [&](int g) { return bar + 8u * (14 + g); };
    auto p_full = [&](int g) { return bar + 8u * (16 + g); };
    auto o_full = [&](int g) { return bar + 8u * (18 + g); };
    const uint32_t drain = bar + 8u * 20;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(gen + (bar - base) + 8 * 21);
    volatile uint32_t *abort_flag = tmem_slot + 1;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x, kv_head = head / p.kv_share;
    const int row_base = (gridDim.y - 1 - blockIdx.y) * 256;   // the longest rows of all heads first
    // key blocks of the two tiles
    int n_blocks[2];
#pragma unroll
    for (int g = 0; g < 2; ++g) {
        const int first = row_base + g * 128, last = min(first + 127, p.rows - 1);
        n_blocks[g] = first < p.rows ? (p.pos0 + last) / 128 + 1 : 0;
    }
    const int n_max = max(n_blocks[0], n_blocks[1]);

    if (threadIdx.x == 0) {
        for (int g = 0; g < 2; ++g) {
            ptx::mbar_init(q_full(g), 1);
            ptx::mbar_init(s_full(g), 1);
            ptx::mbar_init(p_full(g), 128);
            ptx::mbar_init(o_full(g), 1);
        }
        for (int s = 0; s < kPrefillMaxStages; ++s) {
            ptx::mbar_init(k_full(s), 1);
            ptx::mbar_init(k_empty(s), 1);
            ptx::mbar_init(v_full(s), 1);
            ptx::mbar_init(v_empty(s), 1);
        }
        ptx::mbar_init(drain, 1);
        *abort_flag = 0u;
        ptx::fence_mbar_init();
        ptx::prefetch_tensormap(&map_q);
        ptx::prefetch_tensormap(&map_kv);
        ptx::prefetch_tensormap(&map_shared);
    }
    if (warp == 1) {
        ptx::tmem_alloc(ptx::smem_u32(tmem_slot), 512);
        ptx::tmem_relinquish();
    }
    ptx::tc_fence_before();
    __syncthreads();
    ptx::tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    // columns: S / P of tile g at 128 g, O of tile g at 256 + 128 g
    grid_dependency_wait();

    if (warp < 4) {
        ptx::reg_dec<56>();
        if (warp == 0 && lane == 0) {
            bool ok = true;
            const int q_col = head * p.q_stride;
            auto load_q = [&](int g) {
                ptx::mbar_arrive_expect_tx(q_full(g), qk_blocks * kPrefillBlock);
                const uint32_t dst = q_base + g * qk_blocks * kPrefillBlock;
                for (int b = 0; b < p.u_blocks; ++b) ptx::tma_load_2d(dst + b * kPrefillBlock, &map_q, q_col / 2 + b * 32, row_base + g * 128, q_full(g));
                for (int b = 0; b < p.r_blocks; ++b)
                    ptx::tma_load_2d(dst + (p.u_blocks + b) * kPrefillBlock, &map_q, (q_col + p.q_rot) / 2 + b * 32, row_base + g * 128, q_full(g));
            };
            if (n_blocks[0]) load_q(0);
            if (n_blocks[1]) load_q(1);
            for (int j = 0; ok && j < n_max; ++j) {
                const int ks = j % p.k_stages, vs = j % p.v_stages;
                if (!bounded_wait(k_empty(ks), ((j / p.k_stages) & 1) ^ 1, abort_flag, p.status, DEV_TIMEOUT_PRODUCER)) { ok = false; break; }
                ptx::mbar_arrive_expect_tx(k_full(ks), qk_blocks * kPrefillBlock);
                const uint32_t kd = k_base + ks * qk_blocks * kPrefillBlock;
                for (int b = 0; b < p.u_blocks; ++b) ptx::tma_load_2d(kd + b * kPrefillBlock, &map_kv, kv_head * p.dim_pad / 2 + b * 32, j * 128, k_full(ks));
                for (int b = 0; b < p.r_blocks; ++b) ptx::tma_load_2d(kd + (p.u_blocks + b) * kPrefillBlock, &map_shared, p.rot_col0 / 2 + b * 32, j * 128, k_full(ks));
                if (!bounded_wait(v_empty(vs), ((j / p.v_stages) & 1) ^ 1, abort_flag, p.status, DEV_TIMEOUT_PRODUCER)) { ok = false; break; }
                ptx::mbar_arrive_expect_tx(v_full(vs), p.v_blocks * kPrefillBlock);
                const uint32_t vd = v_base + vs * p.v_blocks * kPrefillBlock;
                for (int b = 0; b < p.v_blocks; ++b) ptx::tma_load_2d(vd + b * kPrefillBlock, &map_kv, (p.v_col0 + kv_head * p.v_pad) / 2 + b * 32, j * 128, v_full(vs));
            }
        } else if (warp == 1 && lane == 0) {
            constexpr uint32_t idesc_s = ptx::make_idesc_bf16(128, 128, false, false);
            const uint32_t idesc_o = ptx::make_idesc_bf16(128, p.v_pad, false, true);
            auto scores = [&](int g, int j) {
                const uint32_t qa = q_base + g * qk_blocks * kPrefillBlock, ka = k_base + (j % p.k_stages) * qk_blocks * kPrefillBlock;
                uint32_t acc = 0;
                for (int b = 0; b < qk_blocks; ++b) {
                    const int left = b < p.u_blocks ? p.dim_pad - 64 * b : p.rot_pad - 64 * (b - p.u_blocks);
                    for (int k = 0; k < min(left, 64) / 16; ++k) {
                        const uint64_t da = ptx::make_smem_desc(qa + b * kPrefillBlock + k * 32, 16, 1024, ptx::kLayoutSw128);
                        const uint64_t db = ptx::make_smem_desc(ka + b * kPrefillBlock + k * 32, 16, 1024, ptx::kLayoutSw128);
                        ptx::mma_f16_ss(tmem + 128 * g, da, db, idesc_s, acc);
                        acc = 1;
                    }
                }
                ptx::mma_commit(s_full(g));
            };
            auto values = [&](int g, int j) {
                const uint32_t va = v_base + (j % p.v_stages) * p.v_blocks * kPrefillBlock;
                uint32_t acc = j > 0;
#pragma unroll 1
                for (int part = 0; part < 2; ++part)
                    for (int k = 0; k < 8; ++k) {
                        const uint64_t db = ptx::make_smem_desc(va + k * 2048, kPrefillBlock, 1024, ptx::kLayoutSw128);
                        ptx_attn::mma_f16_ts(tmem + 256 + 128 * g, tmem + 128 * g + 32 * (k >> 1) + 8 * (k & 1) + 16 * part, db, idesc_o, acc);
                        acc = 1;
                    }
                if (j + 1 == n_blocks[g]) ptx::mma_commit(o_full(g));
            };
            bool ok = true;
            for (int j = -1; ok && j < n_max; ++j) {
                bool have_k = false;
                for (int g = 0; ok && g < 2; ++g) {
                    if (j >= 0 && j < n_blocks[g]) {
                        const int vs = j % p.v_stages;
                        if (!bounded_wait(v_full(vs), (j / p.v_stages) & 1, abort_flag, p.status, DEV_TIMEOUT_MMA_FULL) ||
                            !bounded_wait(p_full(g), j & 1, abort_flag, p.status, DEV_TIMEOUT_MMA_TMEM)) { ok = false; break; }
                        ptx::tc_fence_after();
                        values(g, j);
                    }
                    if (j + 1 < n_blocks[g]) {
                        const int ks = (j + 1) % p.k_stages;
                        if (!have_k && !bounded_wait(k_full(ks), ((j + 1) / p.k_stages) & 1, abort_flag, p.status, DEV_TIMEOUT_MMA_FULL)) { ok = false; break; }
                        if (j < 0 && !bounded_wait(q_full(g), 0, abort_flag, p.status, DEV_TIMEOUT_MMA_FULL)) { ok = false; break; }
                        have_k = true;
                        ptx::tc_fence_after();
                        scores(g, j + 1);
                    }
                }
                if (ok && j >= 0) ptx::mma_commit(v_empty(j % p.v_stages));
                if (ok && j + 1 < n_max) ptx::mma_commit(k_empty((j + 1) % p.k_stages));
            }
            ptx::mma_commit(drain);
            bounded_wait(drain, 0u, abort_flag, p.status, DEV_TIMEOUT_DRAIN);
        }
        __syncwarp();
    } else {
        ptx::reg_inc<224>();
        const int g = warp >= 8;
        const int quarter = warp & 3;
        const uint32_t lanes = static_cast<uint32_t>(quarter * 32) << 16;
        const uint32_t s_addr = tmem + lanes + 128 * g, o_addr = tmem + lanes + 256 + 128 * g;
        const int row = row_base + g * 128 + quarter * 32 + lane;
        const int last = p.pos0 + row;             // this row's position: keys 0 .. last are visible
        const int blocks = n_blocks[g];
        float ref = -FLT_MAX, sum = 0.0f;          // reference maximum (of s * scale_log2) and sum of weights against it
        bool ok = true;
        for (int j = 0; j < blocks; ++j) {
            if (!bounded_wait(s_full(g), j & 1, abort_flag, p.status, DEV_TIMEOUT_EPILOGUE)) { ok = false; break; }
            ptx::tc_fence_after();
            const bool whole = j * 128 + 127 <= p.pos0 + row_base + g * 128;   // the tile's first row sees all of this block
            const int seen = last - j * 128;                                   // this row: keys 0 .. seen of the block
            // 1. the row's largest score
            bool near_zero = true;   // no score of the warp's rows beyond the cap: tanh is a polynomial
            float top;
            {
                float most[4] = {-FLT_MAX, -FLT_MAX, -FLT_MAX, -FLT_MAX}, widest[4] = {};
                uint32_t r[2][32];
                ptx::tmem_ld_32x32(s_addr, r[0]);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    ptx::tmem_ld_wait();
                    if (c < 3) ptx::tmem_ld_32x32(s_addr + 32 * (c + 1), r[(c + 1) & 1]);
                    if (CAPPED) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) widest[i & 3] = fmaxf(widest[i & 3], fabsf(__uint_as_float(r[c & 1][i])));
                    }
                    if (whole) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) most[i & 3] = fmaxf(most[i & 3], __uint_as_float(r[c & 1][i]));
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i) most[i & 3] = fmaxf(most[i & 3], 32 * c + i <= seen ? __uint_as_float(r[c & 1][i]) : -FLT_MAX);
                    }
                }
                top = fmaxf(fmaxf(most[0], most[1]), fmaxf(most[2], most[3]));
                if (CAPPED) {
                    near_zero = __all_sync(0xffffffffu, fmaxf(fmaxf(widest[0], widest[1]), fmaxf(widest[2], widest[3])) * p.cap_arg <= 1.0f);
                    top = ptx_attn::capped(fmaxf(top, -1e30f) * p.cap_arg, p.cap_log2);
                } else {
                    top = fmaxf(top, -1e30f) * p.scale_log2;
                }
            }
            if (j == 0) {
                ref = top;   // key 0 is visible to every row
            } else {
                const bool grow = top > ref + 8.0f;   // never where the row sees nothing of this block
                if (__any_sync(0xffffffffu, grow)) {
                    // earlier weights refer to the old maximum: scale O (complete: this block's scores come after it) and the sum
                    const float f = grow ? ptx_attn::exp2_approx(ref - top) : 1.0f;
                    if (grow) ref = top;
                    sum *= f;
                    for (int c = 0; c < p.v_pad; c += 32) {
                        uint32_t r[32];
                        ptx::tmem_ld_32x32(o_addr + c, r);
                        ptx::tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * f);
                        ptx_attn::tmem_st_32x32(o_addr + c, r);
                    }
                }
            }
            // 2. the weights: 32 at a time they take the place of their scores, 16 columns of first terms, 16 of second terms
            const uint64_t scale2 = ptx_attn::pack2(CAPPED ? p.cap_arg : p.scale_log2, CAPPED ? p.cap_arg : p.scale_log2), cap2 = ptx_attn::pack2(p.cap_log2, p.cap_log2),
                           minus_ref = ptx_attn::pack2(-ref, -ref);
            uint64_t sums[2] = {0, 0};
#pragma unroll 1
            for (int c = 0; c < 4; ++c) {
                uint32_t r[32], hi[16], lo[16];
                ptx::tmem_ld_32x32(s_addr + 32 * c, r);
                ptx::tmem_ld_wait();
                float x[32];
                if (!CAPPED || near_zero) {
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        const uint64_t v = ptx_attn::pack2(__uint_as_float(r[i]), __uint_as_float(r[i + 1]));
                        ptx_attn::unpack2(CAPPED ? ptx_attn::fma2(ptx_attn::tanh_inner2(ptx_attn::mul2(v, scale2)), cap2, minus_ref) : ptx_attn::fma2(v, scale2, minus_ref), x[i], x[i + 1]);
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i) x[i] = ptx_attn::capped(__uint_as_float(r[i]) * p.cap_arg, p.cap_log2) - ref;
                }
                if (!whole) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (32 * c + i > seen) x[i] = -1e30f;
                }
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float a = ptx_attn::exp2_approx(x[2 * i]), b = ptx_attn::exp2_approx(x[2 * i + 1]);
                    const uint64_t v = ptx_attn::pack2(a, b);
                    sums[i & 1] = ptx_attn::add2(sums[i & 1], v);
                    hi[i] = ptx::pack_bf16x2(a, b);
                    lo[i] = ptx::pack_bf16x2(a - bf16_lo(hi[i]), b - bf16_hi(hi[i]));
                }
                ptx_attn::tmem_st_32x16(s_addr + 32 * c, hi);
                ptx_attn::tmem_st_32x16(s_addr + 32 * c + 16, lo);
            }
            {
                float a, b;
                ptx_attn::unpack2(ptx_attn::add2(sums[0], sums[1]), a, b);
                sum += a + b;
            }
            ptx_attn::tmem_st_wait();
            ptx::tc_fence_before();
            ptx::mbar_arrive(p_full(g));
        }
        if (ok && blocks > 0) {
            ok = bounded_wait(o_full(g), 0, abort_flag, p.status, DEV_TIMEOUT_EPILOGUE);
            ptx::tc_fence_after();
            if (ok) {
                const float inv = 1.0f / sum;
                const bool store = row < p.rows;
                __nv_bfloat16 *dst = p.out + static_cast<long long>(row) * p.ld_out + head * p.vdim;
                const __nv_bfloat16 *gate = p.gate + static_cast<long long>(row) * p.ld_gate + head * p.vdim;
                const bool vec = p.vdim % 8 == 0 && (reinterpret_cast<uintptr_t>(p.gate) & 15) == 0 && p.ld_out % 8 == 0;
                for (int c = 0; c < p.v_pad; c += 32) {
                    uint32_t r[32];
                    ptx::tmem_ld_32x32(o_addr + c, r);
                    ptx::tmem_ld_wait();
                    if (store && vec) {
#pragma unroll
                        for (int q = 0; q < 4; ++q) {
                            if (c + 8 * q >= p.vdim) continue;
                            const uint4 gw = *reinterpret_cast<const uint4 *>(gate + c + 8 * q);
                            const uint32_t gx[4] = {gw.x, gw.y, gw.z, gw.w};
                            uint32_t o[4];
#pragma unroll
                            for (int e = 0; e < 4; ++e)
                                o[e] = ptx::pack_bf16x2(__uint_as_float(r[8 * q + 2 * e]) * inv * sigmoid_f(bf16_lo(gx[e])),
                                                        __uint_as_float(r[8 * q + 2 * e + 1]) * inv * sigmoid_f(bf16_hi(gx[e])));
                            *reinterpret_cast<uint4 *>(dst + c + 8 * q) = make_uint4(o[0], o[1], o[2], o[3]);
                        }
                    } else if (store) {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (c + i < p.vdim) dst[c + i] = __float2bfloat16_rn(__uint_as_float(r[i]) * inv * sigmoid_f(__bfloat162float(gate[c + i])));
                    }
                    __syncwarp();   // the next load of accumulator columns is a warp-wide instruction
                }
            }
        }
    }

    ptx::tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        for (int i = 0; i < 64; ++i) __nanosleep(1000);   // copies still in flight land before the memory is handed on
    }
    __syncthreads();
    if (warp == 1) {
        ptx::tc_fence_after();
        ptx::tmem_dealloc(tmem, 512);
    }
}

}  // namespace dec
}  // namespace gptb200
