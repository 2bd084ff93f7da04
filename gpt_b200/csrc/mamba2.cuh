// Mamba-2 (state-space duality) layers: short causal convolution, step sizes and decays, the recurrence, the gated norm.
//
// A layer's projection row is [z: inner | x: inner | B: groups * state | C: groups * state] in T, its step sizes [heads] in fp32.  In a
// sequence's slot: the convolution's last inputs [2][taps - 1][channels] in T and the state [2][heads][state][vdim] in fp32 (two copies
// each, see StepEntry::parity).  Steps, decays, exponentials, states and their sums are fp32.
#pragma once

#include "decoder_rows.cuh"

namespace gptb200 {
namespace dec {

// A state of [state x vdim] per head; rows of values | state inputs | state outputs: [x: inner | B: groups * state | C: groups * state].
struct RecurrentShape {
    int heads, vdim, state, groups;
    int inner;                  // heads * vdim
    size_t ssm_state;           // offset in the slot: [2][heads][state][vdim] floats
};

struct MambaShape : RecurrentShape {
    int taps, norm_groups;
    int channels;               // inner + 2 * groups * state
    size_t conv_state;          // offset in the slot
};

// Convolution + silu of one channel per thread; blocks beyond the channels compute the step sizes and log-decays.
// xbc [rows][ld_xbc] T; dt, log_decay [rows][heads].
template <typename T>
__global__ void mamba_conv_kernel(T *__restrict__ xbc, int ld_xbc, float *__restrict__ dt, float *__restrict__ log_decay, const T *__restrict__ proj, long long ld_proj,
                                  const float *__restrict__ dt_raw, int ld_dt, const float *__restrict__ taps, const float *__restrict__ conv_b,
                                  const float *__restrict__ dt_bias, const float *__restrict__ a_log, const MambaShape s, const StepEntry *__restrict__ entries,
                                  const int *__restrict__ row_entry, int conv_blocks, int row0)
{
    grid_dependency_wait();
    grid_dependency_launch();
    const int row = row0 + blockIdx.y;
    if (static_cast<int>(blockIdx.x) >= conv_blocks) {
        const int h = (blockIdx.x - conv_blocks) * blockDim.x + threadIdx.x;
        if (h < s.heads) {
            const float step = softplus_f(dt_raw[static_cast<long long>(row) * ld_dt + h] + dt_bias[h]);
            dt[static_cast<long long>(row) * s.heads + h] = step;
            log_decay[static_cast<long long>(row) * s.heads + h] = -expf(a_log[h]) * step;
        }
        return;
    }
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= s.channels) return;
    const StepEntry e = entries[row_entry[row]];
    const int back = s.taps - 1;
    T *state = reinterpret_cast<T *>(e.slot + s.conv_state);
    const T *old = state + static_cast<long long>(e.parity) * back * s.channels;
    const T *in = proj + s.inner + c;
    // input `k` steps before row r (k < taps); before the portion: the sequence's state
    auto input = [&](int r, int k) {
        const int i = r - e.row0 - k;
        return i >= 0 ? in[static_cast<long long>(r - k) * ld_proj] : old[static_cast<long long>(back + i) * s.channels + c];
    };
    float acc = conv_b[c];
    for (int k = s.taps - 1; k >= 0; --k) acc = fmaf(taps[c * s.taps + (back - k)], to_f(input(row, k)), acc);
    xbc[static_cast<long long>(row) * ld_xbc + c] = from_f<T>(silu_t<T>(acc));
    if (row == e.row0 + e.count - 1) {
        T *next = state + static_cast<long long>(e.parity ^ 1) * back * s.channels;
        for (int k = 0; k < back; ++k) next[static_cast<long long>(back - 1 - k) * s.channels + c] = input(row, k);
    }
}

// The recurrence token by token: one block per (head, entry), state in shared memory.  y [rows][inner] fp32.
template <typename T>
__global__ void mamba_scan_kernel(float *__restrict__ y, const T *__restrict__ xbc, int ld_xbc, const float *__restrict__ dt, const float *__restrict__ log_decay,
                                  const float *__restrict__ d_skip, const RecurrentShape s, const StepEntry *__restrict__ entries)
{
    extern __shared__ float sm[];
    const int P = s.vdim, N = s.state, h = blockIdx.x;
    const StepEntry e = entries[blockIdx.y];
    const int lanes = blockDim.x / P;            // threads that share a column (>= 1)
    float *S = sm;                               // [N][P]
    float *part = S + N * P;                     // [lanes][P]
    float *bc = part + lanes * P;                // B [N] | C [N] | x [P]
    grid_dependency_wait();
    grid_dependency_launch();
    float *state = reinterpret_cast<float *>(e.slot + s.ssm_state) + static_cast<long long>(h) * N * P;
    const float *old_state = state + static_cast<long long>(e.parity) * s.heads * N * P;
    state += static_cast<long long>(e.parity ^ 1) * s.heads * N * P;
    for (int i = threadIdx.x; i < N * P; i += blockDim.x) S[i] = old_state[i];
    const int g = h / (s.heads / s.groups);
    const int p = threadIdx.x % P, q = threadIdx.x / P;
    const bool busy = q < lanes;
    for (int t = 0; t < e.count; ++t) {
        const int row = e.row0 + t;
        const T *src = xbc + static_cast<long long>(row) * ld_xbc;
        __syncthreads();
        for (int i = threadIdx.x; i < N; i += blockDim.x) {
            bc[i] = to_f(src[s.inner + g * N + i]);
            bc[N + i] = to_f(src[s.inner + s.groups * N + g * N + i]);
        }
        for (int i = threadIdx.x; i < P; i += blockDim.x) bc[2 * N + i] = to_f(src[h * P + i]);
        __syncthreads();
        const float step = dt[static_cast<long long>(row) * s.heads + h], keep = expf(log_decay[static_cast<long long>(row) * s.heads + h]);
        if (busy) {
            const float x = bc[2 * N + p];
            float acc = 0.0f;
            for (int n = q; n < N; n += lanes) {
                const float v = fmaf(keep, S[n * P + p], step * bc[n] * x);
                S[n * P + p] = v;
                acc = fmaf(bc[N + n], v, acc);
            }
            part[q * P + p] = acc;
        }
        __syncthreads();
        if (threadIdx.x < P) {
            float acc = 0.0f;
            for (int i = 0; i < lanes; ++i) acc += part[i * P + threadIdx.x];
            y[static_cast<long long>(row) * s.inner + h * P + threadIdx.x] = fmaf(d_skip[h], bc[2 * N + threadIdx.x], acc);
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < N * P; i += blockDim.x) state[i] = S[i];
}

__device__ __forceinline__ void load8(const __nv_bfloat16 *src, uint32_t (&w)[8])   // raw: 8 values in 4 words
{
    const uint4 v = *reinterpret_cast<const uint4 *>(src);
    w[0] = v.x; w[1] = v.y; w[2] = v.z; w[3] = v.w;
}
__device__ __forceinline__ void load8(const float *src, uint32_t (&w)[8])
{
    const uint4 a = *reinterpret_cast<const uint4 *>(src), b = *reinterpret_cast<const uint4 *>(src + 4);
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
}
template <typename T> __device__ __forceinline__ float raw8(const uint32_t (&w)[8], int i);
template <> __device__ __forceinline__ float raw8<float>(const uint32_t (&w)[8], int i) { return __uint_as_float(w[i]); }
template <> __device__ __forceinline__ float raw8<__nv_bfloat16>(const uint32_t (&w)[8], int i) { return i & 1 ? bf16_hi(w[i >> 1]) : bf16_lo(w[i >> 1]); }
__device__ __forceinline__ void store8(__nv_bfloat16 *dst, const float (&v)[8])
{
    *reinterpret_cast<uint4 *>(dst) = make_uint4(ptx::pack_bf16x2(v[0], v[1]), ptx::pack_bf16x2(v[2], v[3]), ptx::pack_bf16x2(v[4], v[5]), ptx::pack_bf16x2(v[6], v[7]));
}
__device__ __forceinline__ void store8(float *dst, const float (&v)[8])
{
    store4(dst, make_float4(v[0], v[1], v[2], v[3]));
    store4(dst + 4, make_float4(v[4], v[5], v[6], v[7]));
}

constexpr int kConvRows = 8;   // consecutive rows per thread

// mamba_conv_kernel for channel counts and offsets that are multiples of 8: a thread slides over eight rows of eight channels with the
// last inputs in registers.  taps_t [taps][channels].
template <typename T, int TAPS>
__global__ void __launch_bounds__(128, 4)
mamba_conv8_kernel(T *__restrict__ xbc, int ld_xbc, float *__restrict__ dt, float *__restrict__ log_decay, const T *__restrict__ proj, long long ld_proj, const float *__restrict__ dt_raw,
                   int ld_dt, const float *__restrict__ taps_t, const float *__restrict__ conv_b, const float *__restrict__ dt_bias, const float *__restrict__ a_log, const MambaShape s,
                   const StepEntry *__restrict__ entries, const int *__restrict__ row_entry, int conv_blocks, int row0, int rows)
{
    constexpr int BACK = TAPS - 1;
    grid_dependency_wait();
    grid_dependency_launch();
    const int first = row0 + blockIdx.y * kConvRows, end = min(first + kConvRows, row0 + rows);
    if (static_cast<int>(blockIdx.x) >= conv_blocks) {
        for (int i = threadIdx.x; i < (end - first) * s.heads; i += blockDim.x) {
            const long long row = first + i / s.heads;
            const int h = i % s.heads;
            const float step = softplus_f(dt_raw[row * ld_dt + h] + dt_bias[h]);
            dt[row * s.heads + h] = step;
            log_decay[row * s.heads + h] = -expf(a_log[h]) * step;
        }
        return;
    }
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    if (c >= s.channels) return;
    uint32_t in[kConvRows][8], window[BACK > 0 ? BACK : 1][8];   // window[k]: the input BACK - k steps back
    const T *src = proj + s.inner + c;
#pragma unroll
    for (int i = 0; i < kConvRows; ++i)
        if (first + i < end) load8(src + static_cast<long long>(first + i) * ld_proj, in[i]);
    float w[TAPS][8], bias[8];
    auto vec8 = [&](const float *from, float (&to)[8]) {
        const float4 a = __ldg(reinterpret_cast<const float4 *>(from)), b = __ldg(reinterpret_cast<const float4 *>(from + 4));
        to[0] = a.x; to[1] = a.y; to[2] = a.z; to[3] = a.w; to[4] = b.x; to[5] = b.y; to[6] = b.z; to[7] = b.w;
    };
    vec8(conv_b + c, bias);
#pragma unroll
    for (int k = 0; k < TAPS; ++k) vec8(taps_t + static_cast<long long>(k) * s.channels + c, w[k]);
    int entry = row_entry[first];
    StepEntry e = entries[entry];
    auto load_window = [&](int row) {   // the inputs before `row`
        const T *old = reinterpret_cast<const T *>(e.slot + s.conv_state) + static_cast<long long>(e.parity) * BACK * s.channels + c;
#pragma unroll
        for (int k = 0; k < BACK; ++k) {
            const int r = row - (BACK - k);
            load8(r >= e.row0 ? src + static_cast<long long>(r) * ld_proj : old + static_cast<long long>(BACK + r - e.row0) * s.channels, window[k]);
        }
    };
    load_window(first);
#pragma unroll
    for (int i = 0; i < kConvRows; ++i) {
        const int row = first + i;
        if (row >= end) break;
        if (row == e.row0 + e.count) {
            e = entries[++entry];
            load_window(row);
        }
        float out[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            float acc = bias[j];
#pragma unroll
            for (int k = 0; k < BACK; ++k) acc = fmaf(w[k][j], raw8<T>(window[k], j), acc);
            out[j] = silu_t<T>(fmaf(w[BACK][j], raw8<T>(in[i], j), acc));
        }
        store8(xbc + static_cast<long long>(row) * ld_xbc + c, out);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
#pragma unroll
            for (int k = 0; k + 1 < BACK; ++k) window[k][j] = window[k + 1][j];
            if (BACK > 0) window[BACK > 0 ? BACK - 1 : 0][j] = in[i][j];
        }
        if (row == e.row0 + e.count - 1) {
            T *next = reinterpret_cast<T *>(e.slot + s.conv_state) + static_cast<long long>(e.parity ^ 1) * BACK * s.channels + c;
#pragma unroll
            for (int k = 0; k < BACK; ++k) {
                float v[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] = raw8<T>(window[k], j);
                store8(next + static_cast<long long>(k) * s.channels, v);
            }
        }
    }
}

constexpr int kStepCols = 32;   // value columns per block of the single-token kernel

// One token: convolution, step size and recurrence in one launch.  One block per (head, 32 value columns, entry): a lane per column,
// the eight warps share the state rows.  The convolution of B and C is computed by every block of the group; its inputs are
// stored by the group's first.
template <typename T>
__global__ void __launch_bounds__(256)
mamba_step_kernel(float *__restrict__ y, const T *__restrict__ proj, long long ld_proj, const float *__restrict__ dt_raw, int ld_dt, const float *__restrict__ taps,
                  const float *__restrict__ conv_b, const float *__restrict__ dt_bias, const float *__restrict__ a_log, const float *__restrict__ d_skip, const MambaShape s,
                  const StepEntry *__restrict__ entries)
{
    extern __shared__ float sm[];   // B [N] | C [N] | x [32] | partial sums [8][32]
    const int P = s.vdim, N = s.state;
    const int slices = (P + kStepCols - 1) / kStepCols;
    const int h = blockIdx.x / slices, p0 = (blockIdx.x % slices) * kStepCols;
    const int per_group = s.heads / s.groups, g = h / per_group;
    float *x = sm + 2 * N, *part = x + kStepCols;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    grid_dependency_wait();
    grid_dependency_launch();
    const StepEntry e = entries[blockIdx.y];
    const long long row = e.row0;
    const int back = s.taps - 1;
    T *conv = reinterpret_cast<T *>(e.slot + s.conv_state);
    const T *old = conv + static_cast<long long>(e.parity) * back * s.channels;
    T *next = conv + static_cast<long long>(e.parity ^ 1) * back * s.channels;
    const bool owns_bc = p0 == 0 && h == g * per_group;
    for (int i = threadIdx.x; i < 2 * N + kStepCols; i += blockDim.x) {
        const bool is_x = i >= 2 * N;
        if (is_x && p0 + i - 2 * N >= P) {
            x[i - 2 * N] = 0.0f;
            continue;
        }
        const int c = is_x ? h * P + p0 + i - 2 * N : i < N ? s.inner + g * N + i : s.inner + s.groups * N + g * N + i - N;
        const T now = proj[row * ld_proj + s.inner + c];
        float acc = conv_b[c];
        for (int k = 0; k < back; ++k) {
            const T v = old[static_cast<long long>(k) * s.channels + c];
            acc = fmaf(taps[c * s.taps + k], to_f(v), acc);
            if ((is_x || owns_bc) && k > 0) next[static_cast<long long>(k - 1) * s.channels + c] = v;
        }
        if ((is_x || owns_bc) && back > 0) next[static_cast<long long>(back - 1) * s.channels + c] = now;
        acc = fmaf(taps[c * s.taps + back], to_f(now), acc);
        sm[i] = to_f(from_f<T>(silu_t<T>(acc)));   // rounded as the convolution of longer portions leaves it
    }
    const float step = softplus_f(dt_raw[row * ld_dt + h] + dt_bias[h]), keep = expf(-expf(a_log[h]) * step);
    __syncthreads();
    float *state = reinterpret_cast<float *>(e.slot + s.ssm_state) + static_cast<long long>(h) * N * P + p0 + lane;
    const float *old_state = state + static_cast<long long>(e.parity) * s.heads * N * P;
    state += static_cast<long long>(e.parity ^ 1) * s.heads * N * P;
    float acc = 0.0f;
    if (p0 + lane < P) {
        const float xs = step * x[lane];
        for (int n0 = warp; n0 < N; n0 += 64) {   // eight rows in flight
            float v[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = n0 + 8 * i < N ? old_state[static_cast<long long>(n0 + 8 * i) * P] : 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int n = n0 + 8 * i;
                if (n < N) {
                    v[i] = fmaf(keep, v[i], xs * sm[n]);
                    state[static_cast<long long>(n) * P] = v[i];
                    acc = fmaf(sm[N + n], v[i], acc);
                }
            }
        }
    }
    part[warp * kStepCols + lane] = acc;
    __syncthreads();
    if (warp == 0 && p0 + lane < P) {
        float v = d_skip[h] * x[lane];
#pragma unroll
        for (int i = 0; i < 8; ++i) v += part[i * kStepCols + lane];
        y[row * s.inner + h * P + p0 + lane] = v;
    }
}

// y * silu(z), then each of norm_groups parts divided by its own root mean square, times weight, as T [rows][ld_out].
template <typename T>
__global__ void mamba_gated_norm_kernel(T *__restrict__ out, int ld_out, const float *__restrict__ y, const T *__restrict__ proj, long long ld_proj,
                                        const float *__restrict__ weight, const MambaShape s, float eps)
{
    extern __shared__ float sm[];   // [part]
    __shared__ float red[32];
    grid_dependency_wait();
    grid_dependency_launch();
    const long long row = blockIdx.x;
    const int part = s.inner / s.norm_groups, c0 = blockIdx.y * part;
    float ss = 0.0f;
    if (part % 4 == 0) {   // y, z and the output are then aligned to four values
        for (int i = 4 * threadIdx.x; i < part; i += 4 * blockDim.x) {
            const float4 a = load4(y + row * s.inner + c0 + i), z = load4(proj + row * ld_proj + c0 + i);
            const float4 v = make_float4(a.x * silu_t<T>(z.x), a.y * silu_t<T>(z.y), a.z * silu_t<T>(z.z), a.w * silu_t<T>(z.w));
            store4(sm + i, v);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        const float inv = rsqrtf(block_sum(ss, red) / part + eps);
        for (int i = 4 * threadIdx.x; i < part; i += 4 * blockDim.x) {
            const float4 v = load4(sm + i), w = load4(weight + c0 + i);
            store4(out + row * ld_out + c0 + i, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
        }
        return;
    }
    for (int i = threadIdx.x; i < part; i += blockDim.x) {
        const float v = y[row * s.inner + c0 + i] * silu_t<T>(to_f(proj[row * ld_proj + c0 + i]));
        sm[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float inv = rsqrtf(block_sum(ss, red) / part + eps);
    for (int i = threadIdx.x; i < part; i += blockDim.x) out[row * ld_out + c0 + i] = from_f<T>(sm[i] * inv * weight[c0 + i]);
}

}  // namespace dec
}  // namespace gptb200
