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
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[blockIdx.y];
    float *state = reinterpret_cast<float *>(e.slot + s.ssm_state) + static_cast<long long>(h) * N * P + p0 + lane;
    const long long copy = static_cast<long long>(s.heads) * N * P;
    const float *old = state + e.parity * copy;
    float *next = state + (e.parity ^ 1) * copy, *mid = keep_state ? part + 8 * kTokenCols + lane : next;
    const int mid_pitch = keep_state ? kTokenCols : P;
    const float keep = decay[h];
    const bool live = p0 + lane < P;
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
            for (int n0 = warp; n0 < N; n0 += 64) {   // eight rows in flight
                float u[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) u[i] = n0 + 8 * i < N ? src[static_cast<long long>(n0 + 8 * i) * sp] : 0.0f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
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
    return 5 * dim + rank + threads + (keep_state ? dim * dim : 0);
}

// One block per (head, entry).  w2 [heads * dim][w2_pitch], w0 / u / weight [heads * dim].
template <typename T>
__global__ void wkv_tokens_kernel(T *__restrict__ out, int ld_out, const T *__restrict__ proj, const float *__restrict__ low, const T *__restrict__ w2, const float *__restrict__ w0,
                                  const float *__restrict__ u, const float *__restrict__ weight, float eps, const WkvShape s, bool keep_state, const StepEntry *__restrict__ entries)
{
    extern __shared__ float sm[];
    __shared__ float red[32];
    const int D = s.dim, h = blockIdx.x, lanes = blockDim.x / D;   // threads that share a value column (>= 1)
    float *r = sm, *k = r + D, *v = k + D, *w = v + D, *bonus = w + D, *tanh_low = bonus + D, *part = tanh_low + s.rank, *S = part + blockDim.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int p = threadIdx.x % D, q = threadIdx.x / D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) bonus[i] = u[h * D + i];
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[blockIdx.y];
    float *state = reinterpret_cast<float *>(e.slot + s.state) + static_cast<long long>(h) * D * D;
    const long long copy = static_cast<long long>(s.heads) * D * D;
    const float *old = state + e.parity * copy;
    float *next = state + (e.parity ^ 1) * copy, *mid = keep_state ? S : next;
    for (int t = 0; t < e.count; ++t) {
        const long long row = e.row0 + t;
        const T *pr = proj + row * s.ld + h * D;
        __syncthreads();
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            r[i] = to_f(pr[i]);
            k[i] = to_f(pr[s.group + i]);
            v[i] = to_f(pr[2 * s.group + i]);
        }
        for (int i = threadIdx.x; i < s.rank; i += blockDim.x) tanh_low[i] = tanhf(low[row * s.ld_low + i]);
        __syncthreads();
        for (int c = warp; c < D; c += warps) {
            const T *m = w2 + static_cast<long long>(h * D + c) * s.w2_pitch;
            float a = 0.0f;
            for (int j = lane; j < s.rank; j += 32) a = fmaf(to_f(m[j]), tanh_low[j], a);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
            if (lane == 0) w[c] = expf(-expf(a + w0[h * D + c]));
        }
        __syncthreads();
        const float *src = (t == 0 ? old : mid) + p;
        float *dst = (t == e.count - 1 ? next : mid) + p;
        float acc = 0.0f;
        if (q < lanes) {
            const float x = v[p];
            for (int n0 = q; n0 < D; n0 += 8 * lanes) {   // eight rows in flight
                float a[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) a[i] = n0 + i * lanes < D ? src[(n0 + i * lanes) * D] : 0.0f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
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
        if (q == 0) out[row * ld_out + h * D + p] = from_f<T>(o * inv * weight[h * D + p] * silu_f(to_f(pr[3 * s.group + p])));
    }
}

}  // namespace dec
}  // namespace gptb200
