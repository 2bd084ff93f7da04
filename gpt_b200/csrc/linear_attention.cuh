// Linear attention layers token by token: a state of [dim x vdim] per head that decays and receives k v^T.
//
//   lightning   S <- decay S + k v^T, o = S^T q with one constant decay per head.  Projection row [v: heads x vdim | k: heads x dim |
//               q: heads x dim | gate] in T, v, k and q after silu: the layout of RecurrentShape, whose chunked kernel serves prompts.
//   wkv         o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T with a decay w per key channel and token from a low-rank map:
//               w = exp(-exp(W2 tanh(W1 x) + w0)).  Projections r, k, v, gate in groups (WkvShape), W1 x in fp32.  Each head's
//               output is divided by its root mean square, times weight, times silu(gate).
// States live in a sequence's slot as [2][heads][dim][vdim] floats (two copies, see StepEntry::parity).  States, decays and sums are fp32.
#pragma once

#include "mamba2.cuh"

namespace gptb200 {
namespace dec {

constexpr int kTokenCols = 32;   // value columns per block
constexpr int kTokenAhead = 16;  // state values per thread in flight

// Both kernels fetch the state (and weights) of their first token before griddepcontrol.wait: the state was written a whole step
// ago, and so were the entries -- the embedding and the layer's norm lie between, and a kernel of a step starts no earlier than
// the wait of the kernel before it.

__host__ __device__ inline int lightning_smem_floats(int dim, bool keep_state) { return 2 * dim + kTokenCols + 8 * kTokenCols + (keep_state ? dim * kTokenCols : 0); }

// One block per (head, 32 value columns, entry): a lane per column, the eight warps share the state rows.  The first token reads the
// sequence's state, the last one writes it; in between it is in shared memory, or (keep_state false: too large) in its new place.
// y [rows][inner].
template <typename T>
__global__ void __launch_bounds__(256)
lightning_tokens_kernel(float *__restrict__ y, const T *__restrict__ proj, long long ld, const float *__restrict__ decay, const RecurrentShape s, bool keep_state,
                        const StepEntry *__restrict__ entries)
{
    extern __shared__ float sm[];
    const int P = s.vdim, N = s.state, slices = (P + kTokenCols - 1) / kTokenCols;
    const int h = blockIdx.x / slices, p0 = blockIdx.x % slices * kTokenCols;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float *k = sm, *q = k + N, *x = q + N, *part = x + kTokenCols;
    const StepEntry e = entries[blockIdx.y];
    float *state = reinterpret_cast<float *>(e.slot + s.ssm_state) + static_cast<long long>(h) * N * P + p0 + lane;
    const long long copy = static_cast<long long>(s.heads) * N * P;
    const float *old = state + e.parity * copy;
    float *next = state + (e.parity ^ 1) * copy, *mid = keep_state ? part + 8 * kTokenCols + lane : next;
    const int mid_pitch = keep_state ? kTokenCols : P;
    const float keep = decay[h];
    const bool live = p0 + lane < P;
    float head_start[kTokenAhead];
#pragma unroll
    for (int i = 0; i < kTokenAhead; ++i) head_start[i] = live && warp + 8 * i < N ? old[static_cast<long long>(warp + 8 * i) * P] : 0.0f;
    grid_dependency_wait();
    grid_dependency_launch();
    for (int t = 0; t < e.count; ++t) {
        const long long row = e.row0 + t;
        const T *r = proj + row * ld;
        __syncthreads();
        for (int i = threadIdx.x; i < 2 * N + kTokenCols; i += blockDim.x) {
            if (i < 2 * N)
                sm[i] = to_f(r[s.inner + (i < N ? h * N + i : s.heads * N + h * N + i - N)]);
            else
                x[i - 2 * N] = p0 + i - 2 * N < P ? to_f(r[h * P + p0 + i - 2 * N]) : 0.0f;
        }
        __syncthreads();
        const float *src = t == 0 ? old : mid;
        float *dst = t == e.count - 1 ? next : mid;
        const int sp = t == 0 ? P : mid_pitch, dp = t == e.count - 1 ? P : mid_pitch;
        float acc = 0.0f;
        if (live) {
            const float v = x[lane];
            for (int n0 = warp; n0 < N; n0 += 8 * kTokenAhead) {
                float u[kTokenAhead];
#pragma unroll
                for (int i = 0; i < kTokenAhead; ++i) u[i] = t == 0 && n0 == warp ? head_start[i] : n0 + 8 * i < N ? src[static_cast<long long>(n0 + 8 * i) * sp] : 0.0f;
#pragma unroll
                for (int i = 0; i < kTokenAhead; ++i) {
                    const int n = n0 + 8 * i;
                    if (n < N) {
                        u[i] = fmaf(keep, u[i], k[n] * v);
                        dst[static_cast<long long>(n) * dp] = u[i];
                        acc = fmaf(q[n], u[i], acc);
                    }
                }
            }
        }
        part[warp * kTokenCols + lane] = acc;
        __syncthreads();
        if (warp == 0 && live) {
            float v = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) v += part[i * kTokenCols + lane];
            y[row * s.inner + h * P + p0 + lane] = v;
        }
    }
}

struct WkvShape {
    int heads, dim;
    int rank, rank_pad;          // of the decay's map
    int w2_pitch;
    long long group, ld;         // r, k, v, gate of a row start at proj + row * ld + {0, 1, 2, 3} * group
    int ld_low;                  // row pitch of W1 x
    size_t state;                // offset in the slot
};

__host__ __device__ inline int wkv_smem_floats(int dim, int rank, int threads, bool keep_state)
{
    return 7 * dim + (rank + 7) / 8 * 8 + threads + (keep_state ? dim * dim : 0);
}

constexpr int kDecayPieces = 4;   // pieces of eight values of W2 that a thread keeps

// One block per (head, entry).  w2 [heads * dim][w2_pitch], w0 / u / weight [heads * dim].
template <typename T>
__global__ void wkv_tokens_kernel(T *__restrict__ out, int ld_out, const T *__restrict__ proj, const float *__restrict__ low, const T *__restrict__ w2, const float *__restrict__ w0,
                                  const float *__restrict__ u, const float *__restrict__ weight, float eps, const WkvShape s, bool keep_state, const StepEntry *__restrict__ entries)
{
    extern __shared__ float sm[];
    __shared__ float red[32];
    const int D = s.dim, h = blockIdx.x, lanes = blockDim.x / D;   // threads that share a value column (>= 1)
    float *tanh_low = sm, *r = tanh_low + s.rank_pad, *k = r + D, *v = k + D, *gate = v + D, *w = gate + D, *bonus = w + D, *part = bonus + D, *S = part + blockDim.x;
    const int p = threadIdx.x % D, q = threadIdx.x / D;
    // the decay's map: `share` neighbouring threads per key channel, eight values at a time
    int share = 32;
    while (share > 1 && share * D > static_cast<int>(blockDim.x)) share >>= 1;
    const int channel = threadIdx.x / share, part_of = threadIdx.x % share;
    const bool maps = channel < D;
    const T *map = w2 + static_cast<long long>(h * D + (maps ? channel : 0)) * s.w2_pitch;
    uint32_t kept[kDecayPieces][8];
#pragma unroll
    for (int i = 0; i < kDecayPieces; ++i)
        if (maps && (part_of + i * share) * 8 < s.rank_pad) load8(map + (part_of + i * share) * 8, kept[i]);
    const float offset = maps ? w0[h * D + channel] : 0.0f, norm_weight = weight[h * D + p];
    for (int i = threadIdx.x; i < D; i += blockDim.x) bonus[i] = u[h * D + i];
    const StepEntry e = entries[blockIdx.y];
    float *state = reinterpret_cast<float *>(e.slot + s.state) + static_cast<long long>(h) * D * D;
    const long long copy = static_cast<long long>(s.heads) * D * D;
    const float *old = state + e.parity * copy;
    float *next = state + (e.parity ^ 1) * copy, *mid = keep_state ? S : next;
    float head_start[kTokenAhead];
#pragma unroll
    for (int i = 0; i < kTokenAhead; ++i) head_start[i] = q < lanes && q + i * lanes < D ? old[(q + i * lanes) * D + p] : 0.0f;
    grid_dependency_wait();
    grid_dependency_launch();
    for (int t = 0; t < e.count; ++t) {
        const long long row = e.row0 + t;
        const T *pr = proj + row * s.ld + h * D;
        __syncthreads();
        for (int i = threadIdx.x; i < 4 * D + s.rank_pad; i += blockDim.x) {   // r, k, v and the gate lie one behind the other in both places
            if (i < 4 * D)
                r[i] = to_f(pr[i / D * s.group + i % D]);
            else
                tanh_low[i - 4 * D] = i - 4 * D < s.rank ? tanhf(low[row * s.ld_low + i - 4 * D]) : 0.0f;
        }
        __syncthreads();
        {
            float a = 0.0f;
            if (maps) {
                auto add = [&](const uint32_t (&m)[8], int at) {
#pragma unroll
                    for (int j = 0; j < 8; ++j) a = fmaf(raw8<T>(m, j), tanh_low[at + j], a);
                };
#pragma unroll
                for (int i = 0; i < kDecayPieces; ++i)
                    if ((part_of + i * share) * 8 < s.rank_pad) add(kept[i], (part_of + i * share) * 8);
                for (int at = (part_of + kDecayPieces * share) * 8; at < s.rank_pad; at += share * 8) {
                    uint32_t m[8];
                    load8(map + at, m);
                    add(m, at);
                }
            }
            for (int o = share >> 1; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
            if (maps && part_of == 0) w[channel] = expf(-expf(a + offset));
        }
        __syncthreads();
        const float *src = (t == 0 ? old : mid) + p;
        float *dst = (t == e.count - 1 ? next : mid) + p;
        float acc = 0.0f;
        if (q < lanes) {
            const float x = v[p];
            for (int n0 = q; n0 < D; n0 += kTokenAhead * lanes) {
                float a[kTokenAhead];
#pragma unroll
                for (int i = 0; i < kTokenAhead; ++i) a[i] = t == 0 && n0 == q ? head_start[i] : n0 + i * lanes < D ? src[(n0 + i * lanes) * D] : 0.0f;
#pragma unroll
                for (int i = 0; i < kTokenAhead; ++i) {
                    const int n = n0 + i * lanes;
                    if (n < D) {
                        const float kv = k[n] * x;
                        acc = fmaf(r[n], fmaf(bonus[n], kv, a[i]), acc);
                        dst[n * D] = fmaf(w[n], a[i], kv);
                    }
                }
            }
        }
        part[threadIdx.x] = acc;
        __syncthreads();
        float o = 0.0f;
        if (q == 0)
            for (int i = 0; i < lanes; ++i) o += part[i * D + p];
        const float inv = rsqrtf(block_sum(o * o, red) / D + eps);
        if (q == 0) out[row * ld_out + h * D + p] = from_f<T>(o * inv * norm_weight * silu_f(gate[p]));
    }
}

}  // namespace dec
}  // namespace gptb200
