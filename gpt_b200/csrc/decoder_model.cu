// DecoderModel: host-side driver of the decoder models described by a config.json (decoder_config.h): weights, sequence states, one
// step over any mixture of requests, sampling, generation.
//
// A step takes, for each of its requests, the next tokens (a prompt, a portion of one, or a single token) and runs only those: what
// came before is in the request's slot -- cached latents or keys and values of the attention layers, convolution inputs and states of
// the recurrent layers, the previous token and its normed residual of the layers that look back at it.  A slot belongs to one request from open to close and
// is zeroed when it is opened.
//
// T is the type of weights, activations and caches: bf16 (products on the tensor cores, or streamed weights for a few rows) or
// float (fp32 FMAs everywhere).  Residual stream, norms, softmax, recurrences and their inputs are fp32 in both.
#include <cstdio>
#include <cstring>
#include <functional>
#include <memory>
#include <type_traits>
#include <vector>

#include "attention_prefill_sm100.cuh"
#include "ctx_internal.h"
#include "decoder_config.h"
#include "decoder_rows.cuh"
#include "grouped_attention.cuh"
#include "latent_attention.cuh"
#include "latent_decode.cuh"
#include "linear_attention.cuh"
#include "mamba2.cuh"
#include "mamba2_chunk.cuh"
#include "safetensors.h"
#include "wkv_chunk.cuh"

using namespace gptb200;
using namespace gptb200::dec;

namespace {

#define RC_TRY(expr)                       \
    do {                                   \
        const int rc_ = (expr);            \
        if (rc_ != GPTB200_OK) return rc_; \
    } while (0)

constexpr int pad_to(int n, int m) { return (n + m - 1) / m * m; }

class DecoderBase
{
public:
    DecoderBase(gptb200_ctx *ctx, const DecoderConfig &c) : ctx_(ctx), c_(c) {}
    virtual ~DecoderBase() = default;
    virtual int load(const SafeTensors &file) = 0;
    virtual int open(int max_len, int *slot) = 0;
    virtual int close(int slot) = 0;
    virtual int length(int slot) const = 0;
    virtual int step(int n, const int *slots, const int *counts, const int *tokens, int n_want, const int *want, float *logits) = 0;
    virtual int generate(int n, const int *slots, const int *first, int steps, float temperature, unsigned long long seed, int *out) = 0;
    virtual int set_option(const char *key, int value) = 0;
    const DecoderConfig &config() const { return c_; }

protected:
    gptb200_ctx *ctx_;
    DecoderConfig c_;
};

template <typename T>
class DecoderModel final : public DecoderBase
{
    static constexpr bool kF32 = std::is_same<T, float>::value;

public:
    using DecoderBase::DecoderBase;

    ~DecoderModel() override
    {
        cudaStreamSynchronize(ctx_->stream);
        drop_graph();
        for (Slot &s : slots_)
            if (s.base) cudaFree(s.base);
        for (void *p : weights_) cudaFree(p);
        for (void *p : work_) cudaFree(p);
        if (expanded_) cudaFree(expanded_);
        if (scratch_) cudaFree(scratch_);
        if (host_) cudaFreeHost(host_);
    }

    // ------------------------------------------------------------------------------------------------ weights
    int load(const SafeTensors &file) override
    {
        pitch_ = pad_to(c_.width, 8);
        vocab_pitch_ = pad_to(c_.vocab, 8);
        side_pitch_ = pad_to(std::max(c_.side_dim, 1), 8);
        const int W = c_.width;
        layers_.resize(c_.layers.size());
        size_t off = 0;
        const auto take = [&](size_t bytes) { const size_t at = off; off += (bytes + 255) & ~size_t(255); return at; };
        RC_TRY(matrix(file, &embed_, {{"embed", c_.vocab}}, W, c_.vocab, pitch_));
        if (c_.pair_buckets > 0) {
            RC_TRY(matrix(file, &pairs_, {{"bigram", static_cast<int>(c_.pair_buckets) + 1}}, W, static_cast<int>(c_.pair_buckets) + 1, pitch_));
            previous_state_ = take(2 * sizeof(int));
        }
        const TensorView *side = c_.traits.token_side ? &tensor(file, "side.embed", {c_.vocab, static_cast<long long>(c_.layers.size()) * c_.side_dim}) : nullptr;
        for (size_t i = 0; i < layers_.size(); ++i) {
            const LayerConfig &l = c_.layers[i];
            Layer &d = layers_[i];
            const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
            RC_TRY(norm(file, &d.norm1, p + "norm1"));
            if (norms_around()) RC_TRY(norm(file, &d.norm1b, p + "norm1b"));
            if (c_.traits.token_shift) {
                RC_TRY(vector(file, &d.shift, p + "shift", W, pitch_));
                d.shift_state = take(2 * size_t(pitch_) * sizeof(float));
            }
            if (c_.traits.depth_average) RC_TRY(vector(file, &d.dwa, p + "dwa", static_cast<int>(i) + 2));
            if (l.kind == MixerKind::Mamba2) {
                const Mamba2Config &a = l.mamba;
                MambaShape &s = d.mamba;
                s = {{a.heads, a.vdim, a.state, a.groups, a.inner(), 0}, a.conv, a.norm_groups, a.conv_channels(), 0};
                d.proj_cols = pad_to(a.inner() + s.channels, 32);      // T columns; the step sizes follow
                d.proj_n = d.proj_cols + pad_to(a.heads, 8);
                const int rows = a.inner() + s.channels;
                RC_TRY(matrix(file, &d.w_in, {{m + "in", rows + a.heads}}, W, d.proj_n, pitch_, [&](int r) { return r < rows ? r : d.proj_cols + r - rows; }));
                RC_TRY(vector(file, &d.taps, m + "conv", s.channels * s.taps, 0, {s.channels, s.taps}));
                RC_TRY(transposed(file, &d.taps_t, m + "conv", s.channels, s.taps));
                RC_TRY(vector(file, &d.conv_b, m + "conv.b", s.channels));
                RC_TRY(vector(file, &d.dt_bias, m + "dt_bias", a.heads));
                RC_TRY(vector(file, &d.a_log, m + "A_log", a.heads));
                RC_TRY(vector(file, &d.d_skip, m + "D", a.heads));
                RC_TRY(vector(file, &d.mix_norm, m + "norm", s.inner));
                d.mix_out = pad_to(s.inner, 8);
                RC_TRY(matrix(file, &d.w_o, {{m + "o", W}}, s.inner, pitch_, d.mix_out));
                s.conv_state = take(2 * size_t(s.taps - 1) * s.channels * sizeof(T));
                s.ssm_state = take(2 * size_t(a.heads) * a.state * a.vdim * sizeof(float));
            } else if (l.kind == MixerKind::Grouped) {
                RC_TRY(load_grouped(file, d, l.grouped, m));
            } else if (l.kind == MixerKind::Lightning) {
                RC_TRY(load_lightning(file, d, l.lightning, m, take));
            } else if (l.kind == MixerKind::Wkv) {
                RC_TRY(load_wkv(file, d, l.wkv, m, take));
            } else {
                const LatentConfig &a = l.latent;
                LatentShape &s = d.latent;
                s = {a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, pad_to(a.kv_rank, 16), pad_to(a.kv_rank, 16) + pad_to(a.rot_dim, 16), pad_to(a.dim, 16), pad_to(a.vdim, 16),
                     pad_to(a.dim, 16) + pad_to(a.rot_dim, 16), a.rot.dims / 2, 0, 0, static_cast<float>(a.scale), 0, 0};
                d.own_keys = a.kv_from < 0;
                const int nq = a.heads * (a.dim + a.rot_dim), nd = d.own_keys ? a.kv_rank + a.rot_dim : 0, ng = a.heads * a.vdim;
                s.off_dkv = a.heads * s.q_stride;
                s.off_g = s.off_dkv + pad_to(nd, 8);
                d.proj_n = d.proj_cols = pad_to(s.off_g + ng, 8);
                std::vector<Piece> pieces = {{m + "q", nq}};
                if (d.own_keys) pieces.push_back({m + "dkv", nd});
                pieces.push_back({m + "g", ng});
                const auto query_row = [&](int r) {
                    const int h = r / (a.dim + a.rot_dim), i = r % (a.dim + a.rot_dim);
                    return h * s.q_stride + (i < a.dim ? i : s.dim_pad + i - a.dim);
                };
                RC_TRY(matrix(file, &d.w_in, pieces, W, d.proj_n, pitch_, [&](int r) { return r < nq ? query_row(r) : r < nq + nd ? s.off_dkv + r - nq : s.off_g + r - nq - nd; }));
                if (d.own_keys) RC_TRY(vector(file, &d.mix_norm, m + "dkv.norm", a.kv_rank));
                RC_TRY(matrix(file, &d.w_uk, {{m + "uk", a.heads * a.dim}, {m + "uv", a.heads * a.vdim}}, a.kv_rank, a.heads * (s.dim_pad + s.v_pad), s.rank_pitch, [&](int r) {
                    const int v = r - a.heads * a.dim;
                    return v < 0 ? r / a.dim * s.dim_pad + r % a.dim : a.heads * s.dim_pad + v / a.vdim * s.v_pad + v % a.vdim;
                }));
                d.w_uv = d.w_uk + size_t(a.heads) * s.dim_pad * s.rank_pitch;
                d.mix_out = pad_to(ng, 8);
                RC_TRY(matrix(file, &d.w_o, {{m + "o", W}}, ng, pitch_, d.mix_out));
                d.cache_owner = d.own_keys ? static_cast<int>(i) : a.kv_from;
                d.rotary = rotary_index(a.rot);
                if (s.row_pitch > 768) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "latent attention: kv_rank + rot_dim beyond 768");
                if (a.dim > 1024) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "latent attention: dim beyond 1024");
            }
            if (l.ff > 0) {
                RC_TRY(norm(file, &d.norm2, p + "norm2"));
                if (norms_around()) RC_TRY(norm(file, &d.norm2b, p + "norm2b"));
                d.ff = pad_to(l.ff, 32);
                // groups of 32 gate rows | 32 up rows, so that one tile of the product holds both halves of its outputs
                RC_TRY(matrix(file, &d.w_glu, {{p + "mlp.gate", l.ff}, {p + "mlp.up", l.ff}}, W, 2 * d.ff, pitch_,
                              [&](int r) { const int up = r >= l.ff, j = up ? r - l.ff : r; return (j >> 5) * 64 + up * 32 + (j & 31); }));
                RC_TRY(matrix(file, &d.w_down, {{p + "mlp.down", W}}, l.ff, pitch_, d.ff));
            }
            if (side) {
                RC_TRY(matrix(file, &d.side_gate, {{p + "side.gate", c_.side_dim}}, W, side_pitch_, pitch_));
                RC_TRY(matrix(file, &d.side_proj, {{p + "side.proj", W}}, c_.side_dim, pitch_, side_pitch_));
                RC_TRY(vector(file, &d.side_norm, p + "side.norm", W, pitch_));
                RC_TRY(columns(*side, &d.side_embed, c_.vocab, static_cast<long long>(c_.layers.size()) * c_.side_dim, static_cast<long long>(i) * c_.side_dim, c_.side_dim, side_pitch_));
            }
            max_proj_ = std::max(max_proj_, kF32 ? d.proj_n : d.proj_cols);
            max_tail_ = std::max(max_tail_, d.proj_n - d.proj_cols);
            max_act_ = std::max({max_act_, d.mix_out, d.ff, side_pitch_});
            max_ff_ = std::max(max_ff_, d.ff);
            if (l.kind == MixerKind::Mamba2) {
                max_channels_ = std::max(max_channels_, pad_to(d.mamba.channels, 8));
                max_heads_ = std::max(max_heads_, d.mamba.heads);
                max_inner_ = std::max(max_inner_, d.mamba.inner);
            }
            if (l.kind == MixerKind::Lightning) max_inner_ = std::max(max_inner_, d.recurrent.inner);
            if (l.kind == MixerKind::Wkv) {
                mixes_ = kWkvMixes;
                max_raw_ = std::max(max_raw_, pad_to(d.wkv.heads * d.wkv.dim, 8));
                max_low_ = std::max(max_low_, 2 * d.wkv.rank_pad);
            }
            if (l.kind == MixerKind::Grouped && l.grouped.value_mix) first_values_cols_ = d.grouped.kv_heads * d.grouped.v_pad;
        }
        RC_TRY(norm(file, &final_norm_, "final.norm"));
        RC_TRY(matrix(file, &head_, {{"head", c_.vocab}}, W, vocab_pitch_, pitch_));
        fixed_state_ = off;
        for (size_t i = 0; i < layers_.size(); ++i)
            if (layers_[i].own_keys) {
                layers_[i].latent.cache_per_position = position_bytes_;
                position_bytes_ += size_t(layers_[i].latent.row_pitch) * sizeof(T);
            }
        for (Layer &d : layers_)
            if (d.grouped.heads) {
                d.grouped.cache_base = fixed_state_;
                d.grouped.cache_per_position = position_bytes_;
                position_bytes_ += size_t(d.grouped.row_pitch) * sizeof(T);
            }
        for (Layer &d : layers_)
            if (d.cache_owner >= 0) {
                d.latent.cache_base = fixed_state_;
                d.latent.cache_per_position = layers_[d.cache_owner].latent.cache_per_position;
            }
        return GPTB200_OK;
    }

    // ------------------------------------------------------------------------------------------------ sequence states
    int open(int max_len, int *slot) override
    {
        if (max_len <= 0 || !slot) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "open: max_len %d", max_len);
        const size_t need = slot_bytes(max_len);
        int at = -1;
        // a free slot that is large enough, else an unused number
        for (size_t i = 0; i < slots_.size() && at < 0; ++i)
            if (!slots_[i].open && slots_[i].bytes >= need) at = static_cast<int>(i);
        for (size_t i = 0; i < slots_.size() && at < 0; ++i)
            if (!slots_[i].open) at = static_cast<int>(i);
        if (at < 0) {
            at = static_cast<int>(slots_.size());
            slots_.push_back(Slot{});
        }
        Slot &s = slots_[at];
        if (s.bytes < need) {
            void *p = nullptr;
            CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
            drop_graph();
            if (s.base) CUDA_TRY(ctx_, cudaFree(s.base));
            s.base = nullptr;
            s.bytes = 0;
            CUDA_TRY(ctx_, cudaMalloc(&p, need));
            s.base = static_cast<char *>(p);
            s.bytes = need;
        }
        CUDA_TRY(ctx_, cudaMemsetAsync(s.base, 0, need, ctx_->stream));
        s.open = true;
        s.capacity = max_len;
        s.length = 0;
        s.parity = 0;
        *slot = at;
        return GPTB200_OK;
    }

    int close(int slot) override
    {
        if (!valid(slot)) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d is not open", slot);
        slots_[slot].open = false;
        return GPTB200_OK;
    }

    int length(int slot) const override { return valid(slot) ? slots_[slot].length : -1; }

    int set_option(const char *key, int value) override
    {
        if (!strcmp(key, "pass_rows")) {   // most rows of one pass: longer steps are worked through in several
            if (value < 1) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "pass_rows must be positive");
            pass_rows_ = value;
            return GPTB200_OK;
        }
        if (!strcmp(key, "chunk_rows")) {   // recurrent layers: shortest portion that takes the chunked tensor-core form (0x7fffffff: none)
            if (value < 1) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "chunk_rows must be positive");
            chunk_rows_ = value;
            return GPTB200_OK;
        }
        if (!strcmp(key, "segment_tokens")) {   // Mamba-2 and lightning prompts: tokens per segment (a multiple of 64)
            if (value < kChunk || value % kChunk) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "segment_tokens must be a multiple of %d", kChunk);
            segment_tokens_ = value;
            return GPTB200_OK;
        }
        if (!strcmp(key, "wkv_segment_tokens")) {   // wkv prompts: tokens per segment (a multiple of 16; 0: automatic)
            if (value < 0 || value % kWkvChunk) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "wkv_segment_tokens must be a multiple of %d", kWkvChunk);
            wkv_segment_tokens_ = value;
            return GPTB200_OK;
        }
        if (!strcmp(key, "expand_rows")) {   // attention: shortest portion that takes the tensor-core form (0x7fffffff: none)
            if (value < 1) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "expand_rows must be positive");
            expand_rows_ = value;
            return GPTB200_OK;
        }
        return gptb200_ctx_set_option(ctx_, key, value);
    }

    // ------------------------------------------------------------------------------------------------ one step
    int step(int n, const int *slots, const int *counts, const int *tokens, int n_want, const int *want, float *logits) override
    {
        int total = 0;
        for (int i = 0; i < n; ++i) {
            if (!valid(slots[i])) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d is not open", slots[i]);
            for (int j = 0; j < i; ++j)
                if (slots[j] == slots[i]) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d twice in one step", slots[i]);
            if (counts[i] <= 0 || counts[i] > slots_[slots[i]].capacity - slots_[slots[i]].length)
                return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d: %d tokens do not fit (%d of %d held)", slots[i], counts[i], slots_[slots[i]].length, slots_[slots[i]].capacity);
            total += counts[i];
        }
        for (int i = 0; i < total; ++i)
            if (tokens[i] < 0 || tokens[i] >= c_.vocab) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "token %d outside the vocabulary", tokens[i]);
        for (int i = 0; i < n_want; ++i)
            if (want[i] < 0 || want[i] >= total) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "row %d is not in the step", want[i]);
        // passes of at most pass_rows_ rows
        int entry = 0, used = 0, first_row = 0;
        while (first_row < total) {
            std::vector<Part> parts;
            int rows = 0;
            while (entry < n && rows < pass_rows_) {
                const int take = std::min(counts[entry] - used, pass_rows_ - rows);
                parts.push_back({slots[entry], rows, take});
                rows += take;
                used += take;
                if (used == counts[entry]) {
                    ++entry;
                    used = 0;
                }
            }
            std::vector<int> local, where;
            for (int i = 0; i < n_want; ++i)
                if (want[i] >= first_row && want[i] < first_row + rows) {
                    local.push_back(want[i] - first_row);
                    where.push_back(i);
                }
            RC_TRY(pass(parts, tokens + first_row, rows, local));
            for (size_t i = 0; i < where.size();) {   // runs of neighbours in one copy
                size_t j = i + 1;
                while (j < where.size() && where[j] == where[j - 1] + 1) ++j;
                CUDA_TRY(ctx_, cudaMemcpy2DAsync(logits + size_t(where[i]) * c_.vocab, size_t(c_.vocab) * 4, logits_ + i * vocab_pitch_, size_t(vocab_pitch_) * 4, size_t(c_.vocab) * 4,
                                                 j - i, cudaMemcpyDeviceToHost, ctx_->stream));
                i = j;
            }
            first_row += rows;
        }
        return gptb200_ctx_synchronize(ctx_);
    }

    // ------------------------------------------------------------------------------------------------ generation
    // `steps` tokens for each of n sequences: first[i] is the token at sequence i's next position; every step runs one token per
    // sequence and samples the next one on the device.  The step is captured once as a CUDA graph (positions, parities and
    // tokens live in device memory) and replayed.
    int generate(int n, const int *slots, const int *first, int steps, float temperature, unsigned long long seed, int *out) override
    {
        if (n <= 0 || steps <= 0) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "generate: nothing to do");
        if (n > pass_rows_) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "generate: %d sequences in a step of at most %d rows", n, pass_rows_);
        std::vector<Part> parts;
        int longest = 0;
        for (int i = 0; i < n; ++i) {
            if (!valid(slots[i])) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d is not open", slots[i]);
            for (int j = 0; j < i; ++j)
                if (slots[j] == slots[i]) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d twice", slots[i]);
            if (steps > slots_[slots[i]].capacity - slots_[slots[i]].length) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "slot %d: %d more tokens do not fit", slots[i], steps);
            if (first[i] < 0 || first[i] >= c_.vocab) return fail(ctx_, GPTB200_ERR_INVALID_ARG, "token %d outside the vocabulary", first[i]);
            parts.push_back({slots[i], i, 1});
            longest = std::max(longest, slots_[slots[i]].capacity);
        }
        std::vector<int> want(n);
        for (int i = 0; i < n; ++i) want[i] = i;
        RC_TRY(reserve(n, n));
        RC_TRY(reserve_history(n, steps));
        CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
        RC_TRY(upload(parts, first, n, want));
        const GenerateControl control{seed, 0, temperature};
        CUDA_TRY(ctx_, cudaMemcpyAsync(gen_control_, &control, sizeof(control), cudaMemcpyHostToDevice, ctx_->stream));
        const auto body = [&]() -> int {
            generating_ = true;
            const int rc = kernels(parts, n, n);
            generating_ = false;
            RC_TRY(rc);
            RC_TRY(launch(sample_advance_kernel, dim3(n), dim3(512), 0, tokens_, history_, gen_control_, logits_, c_.vocab, vocab_pitch_, entries_));
            return launch(advance_step_kernel, dim3(1), dim3(1), 0, gen_control_);
        };
        const bool reuse = graph_ && graph_n_ == n && graph_len_ == longest && graph_history_ == history_;
        int done = 0;
        if (!reuse) {
            drop_graph();
            RC_TRY(body());   // eager: sets kernel attributes, sizes scratch
            done = 1;
            if (steps > 1) {
                cudaGraph_t g = nullptr;
                CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
                cudaStream_t own = ctx_->stream, cap = nullptr;
                CUDA_TRY(ctx_, cudaStreamCreateWithFlags(&cap, cudaStreamNonBlocking));
                ctx_->stream = cap;   // the caller's stream may be the legacy default stream, which cannot be captured
                cudaError_t ce = cudaStreamBeginCapture(cap, cudaStreamCaptureModeThreadLocal);
                const int rc = ce == cudaSuccess ? body() : GPTB200_ERR_CUDA;
                const cudaError_t ee = ce == cudaSuccess ? cudaStreamEndCapture(cap, &g) : ce;
                ctx_->stream = own;
                cudaStreamDestroy(cap);
                if (rc != GPTB200_OK || ee != cudaSuccess) {
                    if (g) cudaGraphDestroy(g);
                    cudaGetLastError();
                    return rc != GPTB200_OK && ce == cudaSuccess ? rc : fail(ctx_, GPTB200_ERR_CUDA, "capture of the generation step: %s", cudaGetErrorString(ee));
                }
                ce = cudaGraphInstantiate(&graph_, g, 0);
                cudaGraphDestroy(g);
                CUDA_TRY(ctx_, ce);
                graph_n_ = n;
                graph_len_ = longest;
                graph_history_ = history_;
            }
        }
        for (; done < steps; ++done) CUDA_TRY(ctx_, cudaGraphLaunch(graph_, ctx_->stream));
        CUDA_TRY(ctx_, cudaMemcpyAsync(out, history_, size_t(steps) * n * sizeof(int), cudaMemcpyDeviceToHost, ctx_->stream));
        for (int i = 0; i < n; ++i) {
            slots_[slots[i]].length += steps;
            slots_[slots[i]].parity ^= steps & 1;
        }
        return gptb200_ctx_synchronize(ctx_);
    }

private:
    struct Norm { float *w = nullptr, *b = nullptr; };
    struct Layer {
        Norm norm1, norm1b, norm2, norm2b;
        float *shift = nullptr, *dwa = nullptr;
        size_t shift_state = 0;
        T *w_in = nullptr, *w_o = nullptr;
        int proj_n = 0, proj_cols = 0, mix_out = 0;
        MambaShape mamba{};
        float *taps = nullptr, *taps_t = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *d_skip = nullptr, *mix_norm = nullptr;
        LatentShape latent{};
        T *w_uk = nullptr, *w_uv = nullptr;
        GroupedShape grouped{};
        float *bias = nullptr, share = 0.0f;        // of the projections; of the first layer's values (negative: this is that layer)
        bool value_mix = false;
        RecurrentShape recurrent{};
        float *decay = nullptr, *log_decay = nullptr;
        int off_gate = 0;
        WkvShape wkv{};
        int group_cols = 0;
        float *mix = nullptr, *w0 = nullptr, *bonus = nullptr;
        T *w2 = nullptr;
        bool own_keys = false;
        int cache_owner = -1, rotary = -1;
        int ff = 0;
        T *w_glu = nullptr, *w_down = nullptr;
        T *side_gate = nullptr, *side_proj = nullptr, *side_embed = nullptr;
        float *side_norm = nullptr;
    };
    struct Slot {
        char *base = nullptr;
        size_t bytes = 0;
        bool open = false;
        int capacity = 0, length = 0, parity = 0;
    };
    struct Part { int slot, row0, count; };
    struct Piece { std::string name; int rows; };
    struct Rotary { RotaryConfig config; double *freq; double gain; size_t table; };

    static constexpr int kWkvMixes = 5;   // r, k, v, gate, decay

    bool norms_around() const { return c_.traits.norms == NormScheme::LayerNormAround; }
    bool valid(int slot) const { return slot >= 0 && slot < static_cast<int>(slots_.size()) && slots_[slot].open; }

    // ---- weights: host image, then one copy
    const TensorView &tensor(const SafeTensors &f, const std::string &name, std::vector<long long> shape) const
    {
        const TensorView &t = f.get(name);
        if (t.shape != shape) throw std::runtime_error("tensor '" + name + "' has another shape than the configuration gives it");
        if (t.dtype != "BF16" && t.dtype != "F32") throw std::runtime_error("tensor '" + name + "' is " + t.dtype);
        return t;
    }
    static float element(const TensorView &t, long long i)
    {
        if (t.dtype == "F32") {
            float v;
            memcpy(&v, t.data + 4 * i, 4);
            return v;
        }
        uint16_t h;
        memcpy(&h, t.data + 2 * i, 2);
        const uint32_t w = static_cast<uint32_t>(h) << 16;
        float v;
        memcpy(&v, &w, 4);
        return v;
    }
    static void put(float *dst, float v) { *dst = v; }
    static void put(__nv_bfloat16 *dst, float v) { *dst = __float2bfloat16(v); }
    template <typename E>
    int to_device(E **out, const std::vector<E> &host)
    {
        void *p = nullptr;
        CUDA_TRY(ctx_, cudaMalloc(&p, std::max<size_t>(host.size(), 1) * sizeof(E)));
        weights_.push_back(p);
        CUDA_TRY(ctx_, cudaMemcpy(p, host.data(), host.size() * sizeof(E), cudaMemcpyHostToDevice));
        *out = static_cast<E *>(p);
        return GPTB200_OK;
    }
    // The named matrices [rows][cols] one below the other as T [rows_out][pitch], zero elsewhere; place(r): row of the image.
    int matrix(const SafeTensors &f, T **out, const std::vector<Piece> &pieces, int cols, int rows_out, int pitch, std::function<int(int)> place = nullptr)
    {
        std::vector<T> host(size_t(rows_out) * pitch, T(0.0f));
        int r = 0;
        for (const Piece &p : pieces) {
            const TensorView &t = tensor(f, p.name, {p.rows, cols});
            for (int i = 0; i < p.rows; ++i, ++r) {
                T *dst = host.data() + size_t(place ? place(r) : r) * pitch;
                if (!kF32 && t.dtype == "BF16")
                    memcpy(static_cast<void *>(dst), t.data + size_t(i) * cols * 2, size_t(cols) * 2);
                else
                    for (int j = 0; j < cols; ++j) put(dst + j, element(t, 1LL * i * cols + j));
            }
        }
        return to_device(out, host);
    }
    int columns(const TensorView &t, T **out, int rows, long long ld, long long first, int cols, int pitch)
    {
        std::vector<T> host(size_t(rows) * pitch, T(0.0f));
        for (int i = 0; i < rows; ++i)
            for (int j = 0; j < cols; ++j) put(host.data() + size_t(i) * pitch + j, element(t, i * ld + first + j));
        return to_device(out, host);
    }
    int vector(const SafeTensors &f, float **out, const std::string &name, int n, int padded = 0, std::vector<long long> shape = {}, float offset = 0.0f)
    {
        const TensorView &t = tensor(f, name, shape.empty() ? std::vector<long long>{n} : shape);
        std::vector<float> host(std::max(n, padded), 0.0f);
        for (int i = 0; i < n; ++i) host[i] = offset + element(t, i);
        return to_device(out, host);
    }
    int transposed(const SafeTensors &f, float **out, const std::string &name, int rows, int cols)
    {
        const TensorView &t = tensor(f, name, {rows, cols});
        std::vector<float> host(size_t(rows) * cols);
        for (int i = 0; i < rows; ++i)
            for (int j = 0; j < cols; ++j) host[size_t(j) * rows + i] = element(t, 1LL * i * cols + j);
        return to_device(out, host);
    }
    int norm(const SafeTensors &f, Norm *out, const std::string &name)
    {
        RC_TRY(vector(f, &out->w, name, c_.width, pitch_, {}, norms_around() ? 0.0f : 1.0f));
        return norms_around() ? vector(f, &out->b, name + ".b", c_.width, pitch_) : GPTB200_OK;
    }

    // ---- mixers
    int load_grouped(const SafeTensors &file, Layer &d, const GroupedConfig &a, const std::string &m)
    {
        GroupedShape &s = d.grouped;
        s.heads = a.heads; s.kv_heads = a.kv_heads; s.dim = a.dim; s.vdim = a.vdim;
        s.dim_pad = pad_to(a.dim, 16);
        s.v_pad = pad_to(a.vdim, 16);
        s.row_pitch = a.kv_heads * (s.dim_pad + s.v_pad);
        s.off_k = a.heads * s.dim_pad;
        s.off_v = s.off_k + a.kv_heads * s.dim_pad;
        s.off_g = s.off_v + a.kv_heads * s.v_pad;
        s.rot_half = a.rot.dims / 2;
        s.scale = static_cast<float>(a.scale);
        s.softcap = static_cast<float>(a.softcap);
        if (std::max(s.dim_pad, s.v_pad) > 768) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "attention: heads beyond 768");
        const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, ng = a.heads * a.vdim;
        d.proj_n = d.proj_cols = pad_to(s.off_g + ng, 8);
        const auto place = [&](int r) {
            if (r < nq) return r / a.dim * s.dim_pad + r % a.dim;
            if ((r -= nq) < nk) return s.off_k + r / a.dim * s.dim_pad + r % a.dim;
            if ((r -= nk) < nv) return s.off_v + r / a.vdim * s.v_pad + r % a.vdim;
            return s.off_g + r - nv;
        };
        RC_TRY(matrix(file, &d.w_in, {{m + "q", nq}, {m + "k", nk}, {m + "v", nv}, {m + "g", ng}}, c_.width, d.proj_n, pitch_, place));
        std::vector<float> bias(d.proj_n, 0.0f);
        int r = 0;
        for (const Piece &p : {Piece{m + "q.b", nq}, Piece{m + "k.b", nk}, Piece{m + "v.b", nv}}) {
            const TensorView &t = tensor(file, p.name, {p.rows});
            for (int i = 0; i < p.rows; ++i, ++r) bias[place(r)] = element(t, i);
        }
        RC_TRY(to_device(&d.bias, bias));
        d.value_mix = a.value_mix;
        if (a.value_mix) d.share = a.first_values ? -1.0f : scalar(file, m + "vmix");
        d.mix_out = pad_to(ng, 8);
        RC_TRY(matrix(file, &d.w_o, {{m + "o", c_.width}}, ng, pitch_, d.mix_out));
        if (a.rot.dims) d.rotary = rotary_index(a.rot);
        return GPTB200_OK;
    }

    template <typename Take>
    int load_lightning(const SafeTensors &file, Layer &d, const LightningConfig &a, const std::string &m, Take &&take)
    {
        const int nk = a.heads * a.dim, nv = a.heads * a.vdim;
        RecurrentShape &s = d.recurrent;
        s = {a.heads, a.vdim, a.dim, a.heads, nv, 0};
        d.off_gate = pad_to(nv + 2 * nk, 32);
        d.proj_n = d.proj_cols = d.off_gate + pad_to(nv, 8);
        const int before_gate = nv + 2 * nk;
        RC_TRY(matrix(file, &d.w_in, {{m + "v", nv}, {m + "k", nk}, {m + "q", nk}, {m + "g", nv}}, c_.width, d.proj_n, pitch_,
                      [&](int r) { return r < before_gate ? r : d.off_gate + r - before_gate; }));
        RC_TRY(vector(file, &d.mix_norm, m + "norm", nv));
        d.mix_out = pad_to(nv, 8);
        RC_TRY(matrix(file, &d.w_o, {{m + "o", c_.width}}, nv, pitch_, d.mix_out));
        std::vector<float> decay, log_decay;
        for (double x : a.decay) {
            decay.push_back(static_cast<float>(x));
            log_decay.push_back(static_cast<float>(std::max(std::log(x), -200.0)));   // nothing is left of a value after that
        }
        RC_TRY(to_device(&d.decay, decay));
        RC_TRY(to_device(&d.log_decay, log_decay));
        s.ssm_state = take(2 * size_t(a.heads) * a.dim * a.vdim * sizeof(float));
        return GPTB200_OK;
    }

    template <typename Take>
    int load_wkv(const SafeTensors &file, Layer &d, const WkvConfig &a, const std::string &m, Take &&take)
    {
        const int n = a.heads * a.dim, W = c_.width;
        if (a.dim > 1024) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "wkv: dim beyond 1024");
        const TensorView &w1 = file.get(m + "w1");   // its shape gives the rank
        if (w1.shape.size() != 2 || w1.shape[0] < 1) throw std::runtime_error("tensor '" + m + "w1' is not a matrix");
        WkvShape &s = d.wkv;
        s.heads = a.heads; s.dim = a.dim;
        s.rank = static_cast<int>(w1.shape[0]);
        s.rank_pad = pad_to(s.rank, 8);
        d.group_cols = pad_to(n, 256);               // whole tiles: each group multiplies rows of its own
        d.proj_cols = 4 * d.group_cols;
        d.proj_n = d.proj_cols + s.rank_pad;
        s.ld_low = s.rank_pad;
        RC_TRY(matrix(file, &d.w_in, {{m + "r", n}, {m + "k", n}, {m + "v", n}, {m + "g", n}, {m + "w1", s.rank}}, W, d.proj_n, pitch_,
                      [&](int r) { return std::min(r / n, 4) * d.group_cols + r - std::min(r / n, 4) * n; }));
        // W2 twice side by side: it multiplies values that come as the sum of two bf16 values
        s.w2_pitch = 2 * s.rank_pad;
        const TensorView &w2 = tensor(file, m + "w2", {n, s.rank});
        std::vector<T> image(size_t(pad_to(n, 8)) * s.w2_pitch, T(0.0f));
        for (int i = 0; i < n; ++i)
            for (int j = 0; j < s.rank; ++j) {
                put(image.data() + size_t(i) * s.w2_pitch + j, element(w2, 1LL * i * s.rank + j));
                put(image.data() + size_t(i) * s.w2_pitch + s.rank_pad + j, element(w2, 1LL * i * s.rank + j));
            }
        RC_TRY(to_device(&d.w2, image));
        RC_TRY(vector(file, &d.w0, m + "w0", n));
        RC_TRY(vector(file, &d.bonus, m + "u", n, 0, {a.heads, a.dim}));
        RC_TRY(vector(file, &d.mix_norm, m + "norm", n));
        std::vector<float> mix;
        for (const char *name : {"r", "k", "v", "g", "w"}) {
            const TensorView &t = tensor(file, m + "mu." + name, {W});
            for (int i = 0; i < pitch_; ++i) mix.push_back(i < W ? element(t, i) : 0.0f);
        }
        RC_TRY(to_device(&d.mix, mix));
        d.mix_out = pad_to(n, 8);
        RC_TRY(matrix(file, &d.w_o, {{m + "o", W}}, n, pitch_, d.mix_out));
        d.shift_state = take(2 * size_t(pitch_) * sizeof(float));
        s.state = take(2 * size_t(n) * a.dim * sizeof(float));
        return GPTB200_OK;
    }
    float scalar(const SafeTensors &f, const std::string &name) const
    {
        const TensorView &t = f.get(name);
        return element(t.shape.empty() ? tensor(f, name, {}) : tensor(f, name, {1}), 0);
    }
    int rotary_index(const RotaryConfig &r)
    {
        for (size_t i = 0; i < rotaries_.size(); ++i)
            if (rotaries_[i].config == r) return static_cast<int>(i);
        Rotary x{r, nullptr, 1.0, 0};
        const std::vector<double> f = rotary_frequencies(r, &x.gain);
        if (to_device(&x.freq, f) != GPTB200_OK) throw std::runtime_error("no memory for a frequency table");
        rotaries_.push_back(x);
        return static_cast<int>(rotaries_.size()) - 1;
    }

    // ---- slots: fixed-size states first, then the cached rows of each layer with keys of its own
    size_t slot_bytes(int len) const { return std::max<size_t>(fixed_state_ + position_bytes_ * len, 256); }

    // ---- workspace
    template <typename E>
    int work(E **out, size_t count)
    {
        void *p = nullptr;
        CUDA_TRY(ctx_, cudaMalloc(&p, std::max<size_t>(count, 1) * sizeof(E)));
        work_.push_back(p);
        CUDA_TRY(ctx_, cudaMemsetAsync(p, 0, std::max<size_t>(count, 1) * sizeof(E), ctx_->stream));   // padding columns are read: keep them finite
        *out = static_cast<E *>(p);
        return GPTB200_OK;
    }
    int reserve(int rows, int wanted)
    {
        if (rows <= rows_ && wanted <= wanted_) return GPTB200_OK;
        CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
        drop_graph();
        for (void *p : work_) cudaFree(p);
        work_.clear();
        history_ = nullptr;
        history_count_ = 0;
        rows_ = wanted_ = 0;
        const size_t R = pad_to(std::max(rows, 8), 8), Q = pad_to(std::max(wanted, 1), 8), P = pitch_;
        state_stride_ = static_cast<long long>(R * P);
        RC_TRY(work(&states_, R * P * (c_.traits.depth_average ? layers_.size() + 1 : 1)));
        RC_TRY(work(&x_[0], R * P));
        RC_TRY(work(&x_[1], R * P));
        RC_TRY(work(&y_, R * P));
        RC_TRY(work(&h_, R * P * std::max(mixes_, 1)));
        RC_TRY(work(&proj_, R * max_proj_));
        RC_TRY(work(&tail_, R * max_tail_));
        RC_TRY(work(&xbc_, R * max_channels_));
        RC_TRY(work(&dt_, R * max_heads_));
        RC_TRY(work(&decay_, R * max_heads_));
        RC_TRY(work(&ssm_y_, R * max_inner_));
        RC_TRY(work(&act_, R * max_act_));
        if (first_values_cols_) RC_TRY(work(&first_values_, R * first_values_cols_));
        if (mixes_) {
            RC_TRY(work(&low_, R * max_low_));
            RC_TRY(work(&raw_, R * max_raw_));
        }
        if (kF32) RC_TRY(work(&glu_, R * 2 * max_ff_));
        RC_TRY(work(&entries_, R));
        RC_TRY(work(&row_entry_, R));
        RC_TRY(work(&tokens_, R));
        RC_TRY(work(&want_, Q));
        RC_TRY(work(&hw_, Q * P));
        RC_TRY(work(&logits_, Q * vocab_pitch_));
        RC_TRY(work(&gen_control_, 1));
        size_t pairs = 0;
        for (Rotary &r : rotaries_) {
            r.table = pairs * R;
            pairs += r.config.dims / 2;
        }
        RC_TRY(work(&table_, R * pairs));
        const size_t host_bytes = R * (sizeof(StepEntry) + 2 * sizeof(int)) + Q * sizeof(int) + 64;
        if (host_) cudaFreeHost(host_);
        host_ = nullptr;
        CUDA_TRY(ctx_, cudaMallocHost(&host_, host_bytes));
        rows_ = static_cast<int>(R);
        wanted_ = static_cast<int>(Q);
        return GPTB200_OK;
    }
    int reserve_history(int n, int steps)
    {
        const size_t count = size_t(n) * steps;
        if (count <= history_count_) return GPTB200_OK;
        CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
        RC_TRY(work(&history_, std::max<size_t>(count, 4096)));
        history_count_ = std::max<size_t>(count, 4096);
        return GPTB200_OK;
    }
    void drop_graph()
    {
        if (graph_) cudaGraphExecDestroy(graph_);
        graph_ = nullptr;
    }

    // Step description to the device.  The pinned image is reused: the caller has waited for the stream.
    int upload(const std::vector<Part> &parts, const int *tokens, int rows, const std::vector<int> &want)
    {
        StepEntry *e = reinterpret_cast<StepEntry *>(host_);
        int *re = reinterpret_cast<int *>(e + rows_), *tk = re + rows_, *wa = tk + rows_;
        for (size_t i = 0; i < parts.size(); ++i) {
            const Slot &s = slots_[parts[i].slot];
            e[i] = {s.base, parts[i].row0, parts[i].count, s.length, s.parity, s.capacity};
            for (int r = 0; r < parts[i].count; ++r) re[parts[i].row0 + r] = static_cast<int>(i);
        }
        memcpy(tk, tokens, size_t(rows) * sizeof(int));
        if (!want.empty()) memcpy(wa, want.data(), want.size() * sizeof(int));
        CUDA_TRY(ctx_, cudaMemcpyAsync(entries_, e, parts.size() * sizeof(StepEntry), cudaMemcpyHostToDevice, ctx_->stream));
        CUDA_TRY(ctx_, cudaMemcpyAsync(row_entry_, re, size_t(rows) * sizeof(int), cudaMemcpyHostToDevice, ctx_->stream));
        CUDA_TRY(ctx_, cudaMemcpyAsync(tokens_, tk, size_t(rows) * sizeof(int), cudaMemcpyHostToDevice, ctx_->stream));
        if (!want.empty()) CUDA_TRY(ctx_, cudaMemcpyAsync(want_, wa, want.size() * sizeof(int), cudaMemcpyHostToDevice, ctx_->stream));
        return GPTB200_OK;
    }

    int pass(const std::vector<Part> &parts, const int *tokens, int rows, const std::vector<int> &want)
    {
        CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));   // the pinned image and the logits of the previous pass are free
        RC_TRY(reserve(rows, static_cast<int>(want.size())));
        RC_TRY(upload(parts, tokens, rows, want));
        RC_TRY(kernels(parts, rows, static_cast<int>(want.size())));
        for (const Part &p : parts) {
            slots_[p.slot].length += p.count;
            slots_[p.slot].parity ^= 1;
        }
        return GPTB200_OK;
    }

    // ---- launches
    template <typename... P, typename... A>
    int launch(void (*kernel)(P...), dim3 grid, dim3 block, size_t smem, A... args)
    {
        const void *key = reinterpret_cast<const void *>(kernel);
        if (smem > 48 * 1024 && !ctx_->configured.count(key)) {
            cudaFuncAttributes fixed{};
            CUDA_TRY(ctx_, cudaFuncGetAttributes(&fixed, kernel));
            CUDA_TRY(ctx_, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - static_cast<int>(fixed.sharedSizeBytes)));
            ctx_->configured.insert(key);
        }
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = grid;
        cfg.blockDim = block;
        cfg.dynamicSmemBytes = smem;
        cfg.stream = ctx_->stream;
        cudaLaunchAttribute attr{};
        attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr.val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = &attr;
        cfg.numAttrs = ctx_->decode_early_launch ? 1 : 0;
        ctx_->launches++;
        CUDA_TRY(ctx_, cudaLaunchKernelEx(&cfg, kernel, static_cast<P>(args)...));
        return GPTB200_OK;
    }

    // out[rows][n] = a[rows][k] . w[n][k]^T in fp32
    int linear_f32(float *out, const T *a, const T *w, int rows, int n, int k)
    {
        if constexpr (kF32) {
            return run_linear_f32(ctx_, out, a, w, rows, n, k);
        } else {
            Bf16Linear c{};
            c.M = rows; c.N = n; c.K = k; c.a = a; c.lda = k; c.w = w; c.out_kind = OUT_F32; c.out = out; c.ldo = n;
            return run_linear_bf16(ctx_, c);
        }
    }

    // threads per row of the stream: with few rows a row is spread wider
    int row_threads(int rows) const { return std::min(rows <= 2 * ctx_->num_sms ? 1024 : 256, std::max(32, pad_to(pitch_ / 4, 32))); }

    int layer_begin(int rows, int layer, const T *h, const int *row_list)
    {
        // layer: the layer that begins; layers_.size(): the final norm over the wanted rows
        const bool final = layer == static_cast<int>(layers_.size());
        LayerBegin<T> b{};
        b.rows = rows; b.width = c_.width; b.pitch = pitch_; b.eps = static_cast<float>(c_.eps);
        b.x_in = layer == 0 ? states_ : x_[(layer - 1) & 1];
        if (layer > 0 && c_.traits.token_side) {
            b.side_y = y_;
            b.side_w = layers_[layer - 1].side_norm;
        }
        b.states = states_; b.state_stride = state_stride_;
        if (layer > 0 && c_.traits.depth_average) {
            b.n_states = layer + 1;
            b.coef = layers_[layer - 1].dwa;
        }
        b.x_out = final ? nullptr : x_[layer & 1];
        const Norm &n = final ? final_norm_ : layers_[layer].norm1;
        b.norm_w = n.w; b.norm_b = n.b;
        if (!final && c_.traits.token_shift) {
            b.shift = layers_[layer].shift;
            b.shift_state = layers_[layer].shift_state;
        }
        b.h = const_cast<T *>(h);
        b.entries = entries_; b.row_entry = row_entry_; b.row_list = row_list;
        b.tile = rows <= 512 || !b.shift ? 1 : rows <= 2048 ? 4 : 8;
        return launch(layer_begin_kernel<T>, dim3((rows + b.tile - 1) / b.tile), dim3(row_threads(rows)), 2 * size_t(pitch_) * sizeof(float), b);
    }

    int mamba(const Layer &d, const std::vector<Part> &parts, int rows)
    {
        const MambaShape &s = d.mamba;
        const float *dt_raw = tail_;
        int ld_dt = d.proj_n - d.proj_cols;
        long long ld = d.proj_cols;
        if constexpr (kF32) {
            RC_TRY(run_linear_f32(ctx_, proj_, h_, d.w_in, rows, d.proj_n, pitch_));
            dt_raw = reinterpret_cast<const float *>(proj_) + d.proj_cols;
            ld = ld_dt = d.proj_n;
        } else {
            Bf16Linear c{};
            c.M = rows; c.N = d.proj_n; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.w_in; c.out_kind = OUT_BF16; c.out = proj_; c.ldo = d.proj_cols;
            c.tail = tail_; c.tail_col = d.proj_cols; c.tail_pitch = ld_dt;
            RC_TRY(run_linear_bf16(ctx_, c));
        }
        // single tokens in one launch; long portions in chunks on the tensor cores, short ones token by token, both behind the
        // convolution kernel; neighbours of a kind together
        const auto kind = [&](const Part &p) { return p.count == 1 ? 0 : !kF32 && s.state <= kChunkMaxState && p.count >= chunk_rows_ ? 2 : 1; };
        for (size_t i = 0, j; i < parts.size(); i = j) {
            const int k = kind(parts[i]);
            for (j = i + 1; j < parts.size() && kind(parts[j]) == k;) ++j;
            const int entry0 = static_cast<int>(i), n = static_cast<int>(j - i), row0 = parts[i].row0, run = parts[j - 1].row0 + parts[j - 1].count - row0;
            if (k == 0) {
                RC_TRY(launch(mamba_step_kernel<T>, dim3(s.heads * ((s.vdim + kStepCols - 1) / kStepCols), n), dim3(256), (2 * size_t(s.state) + 9 * kStepCols) * sizeof(float), ssm_y_, proj_, ld,
                              dt_raw, ld_dt, d.taps, d.conv_b, d.dt_bias, d.a_log, d.d_skip, s, entries_ + entry0));
                continue;
            }
            const int ld_xbc = pad_to(s.channels, 8), conv_blocks = (s.channels + 127) / 128, dt_blocks = (s.heads + 127) / 128;
            if (s.channels % 8 == 0 && s.inner % 8 == 0 && s.taps >= 1 && s.taps <= 4) {
                const auto conv8 = [&](auto kernel) {
                    const int blocks = (s.channels / 8 + 127) / 128;
                    return launch(kernel, dim3(blocks + 1, (run + kConvRows - 1) / kConvRows), dim3(128), 0, xbc_, ld_xbc, dt_, decay_, proj_, ld, dt_raw, ld_dt, d.taps_t, d.conv_b, d.dt_bias,
                                  d.a_log, s, entries_, row_entry_, blocks, row0, run);
                };
                RC_TRY(s.taps == 1 ? conv8(mamba_conv8_kernel<T, 1>) : s.taps == 2 ? conv8(mamba_conv8_kernel<T, 2>) : s.taps == 3 ? conv8(mamba_conv8_kernel<T, 3>)
                                                                                                                                     : conv8(mamba_conv8_kernel<T, 4>));
            } else {
                RC_TRY(launch(mamba_conv_kernel<T>, dim3(conv_blocks + dt_blocks, run), dim3(128), 0, xbc_, ld_xbc, dt_, decay_, proj_, ld, dt_raw, ld_dt, d.taps, d.conv_b, d.dt_bias, d.a_log, s,
                              entries_, row_entry_, conv_blocks, row0));
            }
            RC_TRY(k == 2 ? recurrent_chunks(s, {xbc_, ld_xbc, dt_, decay_, s.heads, d.d_skip}, parts, entry0, n) : mamba_tokens(d, entry0, n, ld_xbc));
        }
        const int part = s.inner / s.norm_groups;
        return launch(mamba_gated_norm_kernel<T>, dim3(rows, s.norm_groups), dim3(std::min(256, pad_to((part + 3) / 4, 32))), size_t(part) * sizeof(float), act_, d.mix_out,
                      static_cast<const float *>(ssm_y_), static_cast<const T *>(proj_), ld, static_cast<const float *>(d.mix_norm), s, static_cast<float>(c_.eps));
    }

    // Inputs of the chunked recurrence: rows of values | state inputs | state outputs (RecurrentShape), steps (null: ones), log-decays,
    // skip (null: none).
    struct ChunkInputs {
        const T *rows;
        int ld;
        const float *steps, *log_decay;
        int ld_decay;
        const float *skip;
    };
    int recurrent_chunks(const RecurrentShape &s, const ChunkInputs &in, const std::vector<Part> &parts, int entry0, int n)
    {
        if constexpr (kF32) {
            return fail(ctx_, GPTB200_ERR_INVALID_ARG, "chunked recurrence in fp32");
        } else {
            // segments that run side by side when a request alone would leave most of its time to one chunk after the other
            int longest = 0;
            for (int i = 0; i < n; ++i) longest = std::max(longest, parts[entry0 + i].count);
            const int blocks = s.heads * ((s.vdim + kChunkCols - 1) / kChunkCols);
            const int tokens = longest > segment_tokens_ + segment_tokens_ / 2 ? segment_tokens_ : pad_to(longest, kChunk);
            const int segments = (longest + tokens - 1) / tokens;
            const size_t smem = size_t(chunk_smem_bytes(s.state));
            float *seg_state = nullptr, *seg_decay = nullptr;
            if (segments > 1) {
                const size_t pieces = size_t(n) * s.heads * segments;
                RC_TRY(scratch(pieces * (size_t(s.state) * s.vdim + 1)));
                seg_state = scratch_;
                seg_decay = scratch_ + pieces * s.state * s.vdim;
                RC_TRY(launch(mamba_chunk_kernel<true>, dim3(blocks, n, segments - 1), dim3(kChunkThreads), smem, ssm_y_, in.rows, in.ld, in.steps, in.log_decay, in.ld_decay, in.skip, s,
                              entries_ + entry0, tokens, segments, seg_state, seg_decay));
            }
            return launch(mamba_chunk_kernel<false>, dim3(blocks, n, segments), dim3(kChunkThreads), smem, ssm_y_, in.rows, in.ld, in.steps, in.log_decay, in.ld_decay, in.skip, s,
                          entries_ + entry0, tokens, segments, seg_state, seg_decay);
        }
    }

    int mamba_tokens(const Layer &d, int entry0, int n, int ld_xbc)
    {
        const MambaShape &s = d.mamba;
        const int threads = std::max(256, pad_to(s.vdim, 32));
        if (threads > 1024) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "mamba2: vdim beyond 1024");
        const size_t smem = (size_t(s.state) * s.vdim + size_t(threads / s.vdim) * s.vdim + 2 * s.state + s.vdim) * sizeof(float);
        if (smem > 227 * 1024) return fail(ctx_, GPTB200_ERR_TOO_LARGE, "mamba2: a head's state does not fit in shared memory");
        return launch(mamba_scan_kernel<T>, dim3(s.heads, n), dim3(threads), smem, ssm_y_, static_cast<const T *>(xbc_), ld_xbc, static_cast<const float *>(dt_),
                      static_cast<const float *>(decay_), static_cast<const float *>(d.d_skip), s, entries_ + entry0);
    }

    template <int NR>
    int latent_rows(const Layer &d, const LatentShape &s, int row0, int rows)
    {
        const size_t smem = (size_t(s.row_pitch) + size_t(kLatentWarps) * s.rank_pitch + 2 * kLatentWarps) * sizeof(float);
        return launch(latent_rows_kernel<T, NR>, dim3(s.heads, rows), dim3(kLatentWarps * 32), smem, act_, d.mix_out, static_cast<const T *>(proj_), static_cast<long long>(d.proj_cols),
                      static_cast<const T *>(d.w_uk), static_cast<const T *>(d.w_uv), s, entries_, row_entry_, row0);
    }

    // positions: most that any of the rows sees (an upper bound)
    int latent_absorbed(const Layer &d, int row0, int rows, int positions)
    {
        const LatentShape &s = d.latent;
        if constexpr (kF32) {
            (void)positions;
            RC_TRY(latent_prepare(d, row0, rows));
            if (s.row_pitch <= 128) return latent_rows<4>(d, s, row0, rows);
            if (s.row_pitch <= 256) return latent_rows<8>(d, s, row0, rows);
            if (s.row_pitch <= 384) return latent_rows<12>(d, s, row0, rows);
            if (s.row_pitch <= 576) return latent_rows<18>(d, s, row0, rows);
            return latent_rows<24>(d, s, row0, rows);
        } else {
            // ranges of positions: enough blocks for the machine, at least two tiles each
            const int groups = (s.heads + 15) / 16;
            int splits = std::max(1, 2 * ctx_->num_sms / (rows * groups));
            splits = std::min({splits, 128, std::max(1, (positions + 2 * kSplitTile - 1) / (2 * kSplitTile))});
            const size_t q_count = size_t(rows) * s.heads * s.row_pitch, o_count = size_t(rows) * s.heads * splits * s.rank_pitch, ml_count = size_t(rows) * s.heads * splits * 2;
            RC_TRY(scratch(q_count + o_count + ml_count));
            float *q = scratch_, *o = q + q_count, *ml = o + o_count;
            const int slices = (s.rank_pitch + kQuerySlice - 1) / kQuerySlice;
            RC_TRY(launch(latent_query_kernel, dim3(s.heads * slices + (d.own_keys ? 1 : 0), rows), dim3(256), 0, q, proj_, d.proj_cols, d.w_uk, table_ + rotaries_[d.rotary].table,
                          d.mix_norm, static_cast<float>(c_.eps), s, entries_, row_entry_, row0));
            RC_TRY(launch(latent_split_kernel, dim3(splits, groups, rows), dim3(kSplitThreads), size_t(split_smem_bytes(s.row_pitch)), o, ml, q, s, entries_, row_entry_, row0));
            return launch(latent_combine_kernel, dim3(s.heads * ((s.vdim + kCombineRows - 1) / kCombineRows), rows), dim3(256), size_t(s.rank_pitch) * sizeof(float), act_, d.mix_out, o, ml,
                          splits, proj_, d.proj_cols, d.w_uv, s, entries_, row_entry_, row0);
        }
    }

    // fp32 scratch of the absorbed form (grown on demand; a captured step keeps its address)
    int scratch(size_t count)
    {
        if (count <= scratch_count_) return GPTB200_OK;
        CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
        drop_graph();
        if (scratch_) CUDA_TRY(ctx_, cudaFree(scratch_));
        scratch_ = nullptr;
        scratch_count_ = 0;
        void *p = nullptr;
        CUDA_TRY(ctx_, cudaMalloc(&p, count * sizeof(float)));
        scratch_ = static_cast<float *>(p);
        scratch_count_ = count;
        return GPTB200_OK;
    }

    // Stages of the tensor-core kernel's rings; 0: its tiles do not fit (large heads), the absorbed form serves any number of rows.
    int prefill_stages(const LatentShape &s, int *v_stages) const { return prefill_stages(s.dim_pad, s.row_pitch - s.rank_pitch, s.v_pad, v_stages); }
    int prefill_stages(int dim_pad, int shared_pad, int v_pad, int *v_stages) const
    {
        const int u = (dim_pad + 63) / 64, r = (shared_pad + 63) / 64, v = (v_pad + 63) / 64;
        if (v_pad > 128) return 0;
        for (const auto &st : {std::pair<int, int>{3, 3}, {2, 2}, {2, 1}, {1, 1}})
            if (prefill_smem_bytes(u, r, v, st.first, st.second) <= 232448) {
                *v_stages = st.second;
                return st.first;
            }
        return 0;
    }

    // Expanded form for one request: keys and values of all its positions, then the tensor-core kernel.
    int latent_expanded(const Layer &d, const Part &part)
    {
        if constexpr (kF32) {
            return latent_absorbed(d, part.row0, part.count, 0);
        } else {
            const LatentShape &s = d.latent;
            const Slot &slot = slots_[part.slot];
            const int positions = slot.length + part.count, cols = s.heads * (s.dim_pad + s.v_pad);
            const size_t need = size_t(positions) * cols;
            if (need > expanded_count_) {
                CUDA_TRY(ctx_, cudaStreamSynchronize(ctx_->stream));
                if (expanded_) CUDA_TRY(ctx_, cudaFree(expanded_));
                expanded_ = nullptr;
                expanded_count_ = 0;
                void *p = nullptr;
                CUDA_TRY(ctx_, cudaMalloc(&p, (need + need / 2) * sizeof(T)));
                expanded_ = static_cast<T *>(p);
                expanded_count_ = need + need / 2;
            }
            const T *cache = reinterpret_cast<const T *>(slot.base + s.cache_base + s.cache_per_position * slot.capacity);
            Bf16Linear c{};
            c.M = positions; c.N = cols; c.K = s.rank_pitch; c.a = cache; c.lda = s.row_pitch; c.w = d.w_uk; c.out_kind = OUT_BF16; c.out = expanded_; c.ldo = cols;
            RC_TRY(run_linear_bf16(ctx_, c));
            CUtensorMap mq, mkv, mc;
            const T *q = proj_ + size_t(part.row0) * d.proj_cols;
            RC_TRY(bf16_operand_map(ctx_, &mq, q, part.count, d.proj_cols, d.proj_cols, 128));
            RC_TRY(bf16_operand_map(ctx_, &mkv, expanded_, positions, cols, cols, 128));
            RC_TRY(bf16_operand_map(ctx_, &mc, cache, positions, s.row_pitch, s.row_pitch, 128));
            PrefillParams p{};
            p.rows = part.count; p.pos0 = slot.length;
            p.heads = s.heads; p.vdim = s.vdim; p.v_pad = s.v_pad;
            p.kv_share = 1;
            p.q_stride = s.q_stride; p.q_rot = s.dim_pad;
            p.dim_pad = s.dim_pad; p.rot_pad = s.row_pitch - s.rank_pitch;
            p.u_blocks = (p.dim_pad + 63) / 64; p.r_blocks = (p.rot_pad + 63) / 64; p.v_blocks = (s.v_pad + 63) / 64;
            p.k_stages = prefill_stages(s, &p.v_stages);
            p.v_col0 = s.heads * s.dim_pad;
            p.rot_col0 = s.rank_pitch;
            p.scale_log2 = static_cast<float>(static_cast<double>(s.scale) * 1.4426950408889634);
            p.out = act_ + size_t(part.row0) * d.mix_out; p.ld_out = d.mix_out;
            p.gate = q + s.off_g; p.ld_gate = d.proj_cols;
            p.status = ctx_->d_status;
            return launch(attention_prefill_kernel<false>, dim3(s.heads, (part.count + 255) / 256), dim3(kPrefillThreads),
                          size_t(prefill_smem_bytes(p.u_blocks, p.r_blocks, p.v_blocks, p.k_stages, p.v_stages)), mq, mkv, mc, p);
        }
    }

    int latent(const Layer &d, const std::vector<Part> &parts, int rows)
    {
        if constexpr (kF32) {
            RC_TRY(run_linear_f32(ctx_, proj_, h_, d.w_in, rows, d.proj_n, pitch_));
        } else {
            Bf16Linear c{};
            c.M = rows; c.N = d.proj_n; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.w_in; c.out_kind = OUT_BF16; c.out = proj_; c.ldo = d.proj_cols;
            RC_TRY(run_linear_bf16(ctx_, c));
        }
        const LatentShape &s = d.latent;
        // long portions one by one in the expanded form, runs of short ones together in the absorbed form
        int v_stages = 0;
        const bool tensor = !kF32 && prefill_stages(s, &v_stages) > 0;
        for (size_t i = 0; i < parts.size();) {
            if (tensor && parts[i].count >= expand_rows_) {
                RC_TRY(latent_prepare(d, parts[i].row0, parts[i].count));
                RC_TRY(latent_expanded(d, parts[i]));
                ++i;
                continue;
            }
            size_t j = i;
            int positions = 0;
            for (; j < parts.size() && !(tensor && parts[j].count >= expand_rows_); ++j) {
                const Slot &slot = slots_[parts[j].slot];
                positions = std::max(positions, generating_ ? slot.capacity : slot.length + parts[j].count);
            }
            RC_TRY(latent_absorbed(d, parts[i].row0, parts[j - 1].row0 + parts[j - 1].count - parts[i].row0, positions));
            i = j;
        }
        return GPTB200_OK;
    }

    int latent_prepare(const Layer &d, int row0, int rows)
    {
        return launch(latent_prepare_kernel<T>, dim3(rows), dim3(128), 0, proj_, d.proj_cols, table_ + rotaries_[d.rotary].table, d.mix_norm, static_cast<float>(c_.eps), d.latent,
                      d.own_keys ? 1 : 0, entries_, row_entry_, row0);
    }

    // ---- grouped attention
    int grouped(const Layer &d, const std::vector<Part> &parts, int rows)
    {
        const GroupedShape &s = d.grouped;
        if constexpr (kF32) {
            RC_TRY(run_linear_f32(ctx_, proj_, h_, d.w_in, rows, d.proj_n, pitch_, d.bias));
        } else {
            Bf16Linear c{};
            c.M = rows; c.N = d.proj_n; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.w_in; c.out_kind = OUT_BF16; c.out = proj_; c.ldo = d.proj_cols;
            c.bias = d.bias;
            RC_TRY(run_linear_bf16(ctx_, c));
        }
        const float2 *table = d.rotary >= 0 ? table_ + rotaries_[d.rotary].table : nullptr;
        RC_TRY(launch(grouped_prepare_kernel<T>, dim3(rows), dim3(256), 0, proj_, d.proj_cols, table, d.value_mix ? first_values_ : nullptr, d.share, s, entries_, row_entry_));
        if constexpr (kF32) {
            const int widest = std::max(s.dim, s.v_pad);
            const auto run = [&](auto kernel) {
                return launch(kernel, dim3(s.heads, rows), dim3(kGroupedWarps * 32), size_t(kGroupedWarps) * s.v_pad * sizeof(float), act_, d.mix_out, static_cast<const T *>(proj_),
                              static_cast<long long>(d.proj_cols), s, entries_, row_entry_);
            };
            if (widest <= 64) return run(grouped_rows_kernel<T, 2>);
            if (widest <= 128) return run(grouped_rows_kernel<T, 4>);
            if (widest <= 256) return run(grouped_rows_kernel<T, 8>);
            return run(grouped_rows_kernel<T, 24>);
        } else {
            // long portions one by one on the tensor cores, runs of short ones together over ranges of positions
            int v_stages = 0;
            const int k_stages = prefill_stages(s.dim_pad, 0, s.v_pad, &v_stages);
            const auto is_long = [&](const Part &p) { return k_stages > 0 && p.count >= expand_rows_; };
            for (size_t i = 0, j; i < parts.size(); i = j) {
                j = i + 1;
                if (is_long(parts[i])) {
                    RC_TRY(grouped_prompt(d, parts[i], k_stages, v_stages));
                    continue;
                }
                int positions = 0;
                for (j = i; j < parts.size() && !is_long(parts[j]); ++j) {
                    const Slot &slot = slots_[parts[j].slot];
                    positions = std::max(positions, generating_ ? slot.capacity : slot.length + parts[j].count);
                }
                RC_TRY(grouped_ranges(d, parts[i].row0, parts[j - 1].row0 + parts[j - 1].count - parts[i].row0, positions));
            }
            return GPTB200_OK;
        }
    }

    // positions: most that any of the rows sees (an upper bound)
    int grouped_ranges(const Layer &d, int row0, int rows, int positions)
    {
        if constexpr (kF32) {
            return GPTB200_OK;
        } else {
            const GroupedShape &s = d.grouped;
            const int share = s.heads / s.kv_heads, head_tiles = (share + 15) / 16, slices = (s.v_pad + kGroupedValues - 1) / kGroupedValues, groups = s.kv_heads * head_tiles * slices;
            constexpr int turn = kGroupedWarps * kGroupedTile;
            int splits = std::max(1, 2 * ctx_->num_sms / (rows * groups));
            splits = std::min({splits, kGroupedMaxSplits, (positions + turn - 1) / turn});
            const size_t o_count = size_t(rows) * s.heads * splits * s.v_pad, ml_count = size_t(rows) * s.heads * splits * 2;
            RC_TRY(scratch(o_count + ml_count));
            float *o = scratch_, *ml = o + o_count;
            const int v_cols = std::min(s.v_pad, kGroupedValues);
            int stages = 4;
            while (stages > 2 && grouped_smem_bytes(s.dim_pad, v_cols, stages) > (stages == 4 ? 110 : 220) * 1024) --stages;
            const auto split = [&](auto kernel) {
                return launch(kernel, dim3(splits, groups, rows), dim3(kGroupedWarps * 32), size_t(grouped_smem_bytes(s.dim_pad, v_cols, stages)), o, ml, proj_, d.proj_cols, s, stages, head_tiles,
                              entries_, row_entry_, row0);
            };
            RC_TRY(v_cols <= 64 ? split(grouped_split_kernel<8>) : split(grouped_split_kernel<16>));
            return launch(grouped_combine_kernel, dim3(s.heads, rows), dim3(kGroupedCombineWarps * 32), size_t(kGroupedCombineWarps) * s.v_pad * sizeof(float), act_, d.mix_out, o, ml, splits, proj_, d.proj_cols, s, entries_, row_entry_, row0);
        }
    }

    int grouped_prompt(const Layer &d, const Part &part, int k_stages, int v_stages)
    {
        if constexpr (kF32) {
            return GPTB200_OK;
        } else {
            const GroupedShape &s = d.grouped;
            const Slot &slot = slots_[part.slot];
            const T *cache = reinterpret_cast<const T *>(slot.base + s.cache_base + s.cache_per_position * slot.capacity), *q = proj_ + size_t(part.row0) * d.proj_cols;
            CUtensorMap mq, mkv;
            RC_TRY(bf16_operand_map(ctx_, &mq, q, part.count, d.proj_cols, d.proj_cols, 128));
            RC_TRY(bf16_operand_map(ctx_, &mkv, cache, slot.length + part.count, s.row_pitch, s.row_pitch, 128));
            PrefillParams p{};
            p.rows = part.count; p.pos0 = slot.length;
            p.heads = s.heads; p.vdim = s.vdim; p.v_pad = s.v_pad;
            p.kv_share = s.heads / s.kv_heads;
            p.q_stride = s.dim_pad; p.q_rot = s.dim_pad;
            p.dim_pad = s.dim_pad; p.rot_pad = 0;
            p.u_blocks = (s.dim_pad + 63) / 64; p.r_blocks = 0; p.v_blocks = (s.v_pad + 63) / 64;
            p.k_stages = k_stages; p.v_stages = v_stages;
            p.v_col0 = s.kv_heads * s.dim_pad;
            constexpr double kLog2e = 1.4426950408889634;
            p.scale_log2 = static_cast<float>(s.scale * kLog2e);
            if (s.softcap > 0.0f) {
                p.cap_log2 = static_cast<float>(s.softcap * kLog2e);
                p.cap_arg = s.scale / s.softcap;
            }
            p.out = act_ + size_t(part.row0) * d.mix_out; p.ld_out = d.mix_out;
            p.gate = q + s.off_g; p.ld_gate = d.proj_cols;
            p.status = ctx_->d_status;
            const size_t smem = size_t(prefill_smem_bytes(p.u_blocks, 0, p.v_blocks, k_stages, v_stages));
            const dim3 grid(s.heads, (part.count + 255) / 256);
            return s.softcap > 0.0f ? launch(attention_prefill_kernel<true>, grid, dim3(kPrefillThreads), smem, mq, mkv, mkv, p)
                                    : launch(attention_prefill_kernel<false>, grid, dim3(kPrefillThreads), smem, mq, mkv, mkv, p);
        }
    }

    // ---- linear attention with constant decays
    int lightning(const Layer &d, const std::vector<Part> &parts, int rows)
    {
        const RecurrentShape &s = d.recurrent;
        if constexpr (kF32) {
            RC_TRY(run_linear_f32(ctx_, proj_, h_, d.w_in, rows, d.proj_n, pitch_));
            RC_TRY(launch(silu_columns_kernel, dim3(rows), dim3(256), 0, proj_, d.off_gate, d.proj_cols));
        } else {
            Bf16Linear c{};
            c.M = rows; c.N = d.proj_n; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.w_in; c.out_kind = OUT_BF16; c.out = proj_; c.ldo = d.proj_cols;
            c.silu_cols = d.off_gate;
            RC_TRY(run_linear_bf16(ctx_, c));
        }
        RC_TRY(runs(parts, [&](const Part &p) { return !kF32 && s.state <= kChunkMaxState && p.count >= chunk_rows_; }, [&](bool chunks, int entry0, int n) {
            if (chunks) return recurrent_chunks(s, {proj_, d.proj_cols, nullptr, d.log_decay, 0, nullptr}, parts, entry0, n);
            const bool keep_state = lightning_smem_floats(s.state, true) * sizeof(float) <= 96 * 1024;
            return launch(lightning_tokens_kernel<T>, dim3(s.heads * ((s.vdim + kTokenCols - 1) / kTokenCols), n), dim3(256), lightning_smem_floats(s.state, keep_state) * sizeof(float), ssm_y_,
                          static_cast<const T *>(proj_), static_cast<long long>(d.proj_cols), static_cast<const float *>(d.decay), s, keep_state, entries_ + entry0);
        }));
        return launch(normed_sigmoid_gate_kernel<T>, dim3(rows), dim3(std::min(1024, pad_to((s.inner + 3) / 4, 32))), size_t(s.inner) * sizeof(float), act_, d.mix_out,
                      static_cast<const float *>(ssm_y_), s.inner, static_cast<const T *>(proj_ + d.off_gate), static_cast<long long>(d.proj_cols), static_cast<const float *>(d.mix_norm),
                      static_cast<float>(c_.eps));
    }

    // Calls run(kind, first part, parts) for every stretch of neighbouring parts of one kind.
    template <typename Kind, typename Run>
    int runs(const std::vector<Part> &parts, Kind &&kind, Run &&run)
    {
        for (size_t i = 0, j; i < parts.size(); i = j) {
            const auto k = kind(parts[i]);
            for (j = i + 1; j < parts.size() && kind(parts[j]) == k;) ++j;
            RC_TRY(run(k, static_cast<int>(i), static_cast<int>(j - i)));
        }
        return GPTB200_OK;
    }

    // ---- wkv: h_ holds the five blends of the normed rows
    int wkv(const Layer &d, const std::vector<Part> &parts, int rows)
    {
        WkvShape s = d.wkv;
        const int n = s.heads * s.dim;
        if constexpr (kF32) {
            s.group = static_cast<long long>(rows) * d.group_cols;
            s.ld = d.group_cols;
            for (int g = 0; g < 5; ++g)
                RC_TRY(run_linear_f32(ctx_, g < 4 ? proj_ + g * s.group : tail_, h_ + g * state_stride_, d.w_in + size_t(g) * d.group_cols * pitch_, rows, g < 4 ? d.group_cols : s.rank_pad, pitch_));
        } else {
            s.group = d.group_cols;
            s.ld = d.proj_cols;
            Bf16Linear c{};
            c.M = rows; c.N = d.proj_n; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.w_in; c.out_kind = OUT_BF16; c.out = proj_; c.ldo = d.proj_cols;
            c.tail = tail_; c.tail_col = d.proj_cols; c.tail_pitch = s.rank_pad;
            c.group_cols = d.group_cols; c.group_rows = rows_;
            RC_TRY(run_linear_bf16(ctx_, c));
        }
        const auto is_long = [&](const Part &p) { return !kF32 && s.dim <= kWkvMaxDim && p.count >= chunk_rows_; };
        if constexpr (!kF32) {
            if (std::any_of(parts.begin(), parts.end(), is_long)) {
                RC_TRY(launch(wkv_low_rank_kernel, dim3(rows), dim3(std::min(128, pad_to(s.rank_pad, 32))), 0, low_, s.rank_pad, tail_, s.ld_low, s.rank));
                Bf16Linear c{};
                c.M = rows; c.N = pad_to(n, 8); c.K = 2 * s.rank_pad; c.a = low_; c.lda = 2 * s.rank_pad; c.w = d.w2; c.out_kind = OUT_F32; c.out = raw_; c.ldo = pad_to(n, 8);
                RC_TRY(run_linear_bf16(ctx_, c));
            }
        }
        return runs(parts, is_long, [&](bool chunks, int entry0, int count) {
            if (chunks) return s.dim <= 32 ? wkv_chunks<2>(d, s, parts, entry0, count) : s.dim <= 64 ? wkv_chunks<4>(d, s, parts, entry0, count) : wkv_chunks<8>(d, s, parts, entry0, count);
            const int threads = std::max(256, pad_to(s.dim, 32));
            const bool keep_state = wkv_smem_floats(s.dim, s.rank, threads, true) * sizeof(float) <= 200 * 1024;
            return launch(wkv_tokens_kernel<T>, dim3(s.heads, count), dim3(threads), wkv_smem_floats(s.dim, s.rank, threads, keep_state) * sizeof(float), act_, d.mix_out,
                          static_cast<const T *>(proj_), static_cast<const float *>(tail_), static_cast<const T *>(d.w2), static_cast<const float *>(d.w0), static_cast<const float *>(d.bonus),
                          static_cast<const float *>(d.mix_norm), static_cast<float>(c_.eps), s, keep_state, entries_ + entry0);
        });
    }

    template <int KT>
    int wkv_chunks(const Layer &d, const WkvShape &s, const std::vector<Part> &parts, int entry0, int n)
    {
        if constexpr (kF32) {
            return GPTB200_OK;
        } else {
            int longest = 0;
            for (int i = 0; i < n; ++i) longest = std::max(longest, parts[entry0 + i].count);
            // segments: as many blocks as fit the machine at once, none shorter than a few chunks
            int segment = wkv_segment_tokens_;
            if (segment == 0) segment = std::max(4 * kWkvChunk, pad_to(static_cast<int>(1LL * longest * n * s.heads / (wkv_blocks(KT) * ctx_->num_sms)), kWkvChunk));
            const int tokens = longest > segment + segment / 2 ? segment : pad_to(longest, kWkvChunk), segments = (longest + tokens - 1) / tokens;
            const size_t smem = wkv_chunk_layout(KT).total, square = size_t(s.dim) * s.dim;
            float *seg_state = nullptr, *seg_decay = nullptr;
            const auto chunks = [&](auto kernel, int launched) {
                return launch(kernel, dim3(s.heads, n, launched), dim3(32 * KT), smem, act_, d.mix_out, proj_, raw_, pad_to(s.heads * s.dim, 8), d.w0, d.bonus, d.mix_norm,
                              static_cast<float>(c_.eps), s, entries_ + entry0, tokens, segments, seg_state, seg_decay);
            };
            if (segments > 1) {
                const size_t pieces = size_t(n) * s.heads * segments;
                RC_TRY(scratch(pieces * (square + s.dim)));
                seg_state = scratch_;
                seg_decay = scratch_ + pieces * square;
                RC_TRY(chunks(wkv_chunk_kernel<KT, true>, segments - 1));
                RC_TRY(launch(wkv_segments_kernel, dim3(s.heads * static_cast<int>((square + 255) / 256), n), dim3(256), 0, seg_state, seg_decay, s, entries_ + entry0, tokens, segments));
            }
            return chunks(wkv_chunk_kernel<KT, false>, segments);
        }
    }

    int mixer(int layer, const std::vector<Part> &parts, int rows)
    {
        const Layer &d = layers_[layer];
        switch (c_.layers[layer].kind) {
            case MixerKind::Mamba2: return mamba(d, parts, rows);
            case MixerKind::Latent: return latent(d, parts, rows);
            case MixerKind::Grouped: return grouped(d, parts, rows);
            case MixerKind::Lightning: return lightning(d, parts, rows);
            default: return wkv(d, parts, rows);
        }
    }

    // y_ = gated feed-forward of h_
    int feed_forward(const Layer &d, int rows)
    {
        if constexpr (kF32) {
            RC_TRY(run_linear_f32(ctx_, glu_, h_, d.w_glu, rows, 2 * d.ff, pitch_));
            RC_TRY(launch(glu_rows_kernel, dim3(rows), dim3(128), 0, act_, static_cast<const float *>(glu_), d.ff, static_cast<long long>(2 * d.ff), c_.traits.silu_gate));
        } else {
            Bf16Linear c{};
            c.M = rows; c.N = 2 * d.ff; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.w_glu; c.out_kind = c_.traits.silu_gate ? OUT_GLU_SILU : OUT_GLU; c.out = act_; c.ldo = d.ff;
            RC_TRY(run_linear_bf16(ctx_, c));
        }
        return linear_f32(y_, act_, d.w_down, rows, pitch_, d.ff);
    }

    // h = norm(x + residual_mult * y), or the layer's blends of it; the sum goes to the other buffer of x_ (`at`: the current one)
    int residual_norm(int rows, int *at, const float *y, const Norm &n, T *h, const Layer *mixes, const int *row_list)
    {
        ResidualNorm<T> b{};
        b.rows = rows; b.width = c_.width; b.pitch = pitch_; b.eps = static_cast<float>(c_.eps); b.mult = static_cast<float>(c_.residual_mult);
        b.x_in = x_[*at];
        b.y = y;
        if (y && !row_list) {
            *at ^= 1;
            b.x_out = x_[*at];
        }
        b.norm_w = n.w;
        if (mixes && mixes->mix) {
            b.mixes = kWkvMixes;
            b.mix = mixes->mix;
            b.shift_state = mixes->shift_state;
            b.mix_stride = state_stride_;
        }
        b.h = h;
        b.entries = entries_; b.row_entry = row_entry_; b.row_list = row_list;
        b.tile = rows <= 512 || !b.mixes ? 1 : rows <= 2048 ? 4 : 8;
        return launch(residual_norm_kernel<T>, dim3((rows + b.tile - 1) / b.tile), dim3(row_threads(rows)), 2 * size_t(pitch_) * sizeof(float), b);
    }

    int rotary_tables(int rows)
    {
        for (const Rotary &r : rotaries_)
            RC_TRY(launch(rotary_table_kernel, dim3((rows * (r.config.dims / 2) + 127) / 128), dim3(128), 0, table_ + r.table, static_cast<const double *>(r.freq), r.config.dims / 2, r.gain,
                          entries_, row_entry_, rows));
        return GPTB200_OK;
    }

    // Norms before the sublayers only: every residual sum happens in the norm that reads it.
    int kernels_norms_before(const std::vector<Part> &parts, int rows, int n_want)
    {
        int at = 0;
        RC_TRY(launch(embed_pair_rows_kernel<T>, dim3(rows), dim3(row_threads(rows)), 0, x_[0], static_cast<const T *>(embed_), static_cast<float>(c_.embed_scale),
                      static_cast<const T *>(pairs_), c_.pair_buckets, c_.pair_mul_previous, c_.pair_mul_current, static_cast<const int *>(tokens_), pitch_, previous_state_, entries_, row_entry_));
        RC_TRY(rotary_tables(rows));
        const float *y = nullptr;
        for (size_t i = 0; i < layers_.size(); ++i) {
            const Layer &d = layers_[i];
            RC_TRY(residual_norm(rows, &at, y, d.norm1, h_, &d, nullptr));
            RC_TRY(mixer(static_cast<int>(i), parts, rows));
            RC_TRY(linear_f32(y_, act_, d.w_o, rows, pitch_, d.mix_out));
            y = y_;
            if (d.ff) {
                RC_TRY(residual_norm(rows, &at, y, d.norm2, h_, nullptr, nullptr));
                RC_TRY(feed_forward(d, rows));
            }
        }
        if (n_want > 0) {
            RC_TRY(residual_norm(n_want, &at, y, final_norm_, hw_, nullptr, want_));
            RC_TRY(linear_f32(logits_, hw_, head_, n_want, vocab_pitch_, pitch_));
        }
        return GPTB200_OK;
    }

    // All kernels of one step; everything that changes from step to step is read from device memory.
    int kernels(const std::vector<Part> &parts, int rows, int n_want)
    {
        if (!norms_around()) return kernels_norms_before(parts, rows, n_want);
        const float eps = static_cast<float>(c_.eps);
        RC_TRY(launch(embed_rows_kernel<T>, dim3(rows), dim3(row_threads(rows)), 0, states_, static_cast<const T *>(embed_), static_cast<const int *>(tokens_), pitch_));
        RC_TRY(rotary_tables(rows));
        for (size_t i = 0; i < layers_.size(); ++i) {
            const Layer &d = layers_[i];
            float *x = x_[i & 1];
            RC_TRY(layer_begin(rows, static_cast<int>(i), h_, nullptr));
            RC_TRY(mixer(static_cast<int>(i), parts, rows));
            RC_TRY(linear_f32(y_, act_, d.w_o, rows, pitch_, d.mix_out));
            const size_t smem = size_t(pitch_) * sizeof(float);
            RC_TRY(launch(sublayer_end_kernel<T>, dim3(rows), dim3(row_threads(rows)), smem, x, static_cast<const float *>(y_), static_cast<const float *>(d.norm1b.w),
                          static_cast<const float *>(d.norm1b.b), static_cast<const float *>(d.norm2.w), static_cast<const float *>(d.norm2.b), h_, c_.width, pitch_, eps));
            if (d.ff) {
                RC_TRY(feed_forward(d, rows));
                RC_TRY(launch(sublayer_end_kernel<T>, dim3(rows), dim3(row_threads(rows)), smem, x, static_cast<const float *>(y_), static_cast<const float *>(d.norm2b.w),
                              static_cast<const float *>(d.norm2b.b), static_cast<const float *>(nullptr), static_cast<const float *>(nullptr), h_, c_.width, pitch_, eps));
            }
            if (d.side_gate) {
                if constexpr (kF32) {
                    RC_TRY(run_linear_f32(ctx_, act_, h_, d.side_gate, rows, side_pitch_, pitch_));
                    RC_TRY(launch(gelu_factor_rows_kernel, dim3(rows), dim3(128), 0, act_, static_cast<const float *>(d.side_embed), static_cast<const int *>(tokens_), side_pitch_));
                } else {
                    Bf16Linear c{};
                    c.M = rows; c.N = side_pitch_; c.K = pitch_; c.a = h_; c.lda = pitch_; c.w = d.side_gate; c.out_kind = OUT_GELU_MUL; c.out = act_; c.ldo = side_pitch_;
                    c.factor = d.side_embed; c.factor_rows = tokens_; c.factor_pitch = side_pitch_;
                    RC_TRY(run_linear_bf16(ctx_, c));
                }
                RC_TRY(linear_f32(y_, act_, d.side_proj, rows, pitch_, side_pitch_));
            }
        }
        if (n_want > 0) {
            RC_TRY(layer_begin(n_want, static_cast<int>(layers_.size()), hw_, want_));
            RC_TRY(linear_f32(logits_, hw_, head_, n_want, vocab_pitch_, pitch_));
        }
        return GPTB200_OK;
    }

    std::vector<Layer> layers_;
    std::vector<Rotary> rotaries_;
    T *embed_ = nullptr, *head_ = nullptr, *pairs_ = nullptr;
    Norm final_norm_;
    int pitch_ = 0, vocab_pitch_ = 0, side_pitch_ = 0;
    int max_proj_ = 8, max_tail_ = 8, max_act_ = 8, max_ff_ = 8, max_channels_ = 8, max_heads_ = 1, max_inner_ = 8;
    int mixes_ = 0, max_raw_ = 0, max_low_ = 0, first_values_cols_ = 0;
    size_t fixed_state_ = 0, position_bytes_ = 0, previous_state_ = 0;
    std::vector<void *> weights_, work_;
    std::vector<Slot> slots_;
    int pass_rows_ = 4096, expand_rows_ = 32, chunk_rows_ = 8, segment_tokens_ = 1024, wkv_segment_tokens_ = 0;
    T *expanded_ = nullptr;
    size_t expanded_count_ = 0;
    float *scratch_ = nullptr;
    size_t scratch_count_ = 0;
    bool generating_ = false;   // launches must serve every length up to the slots' capacities
    int rows_ = 0, wanted_ = 0;
    long long state_stride_ = 0;
    float *states_ = nullptr, *x_[2] = {nullptr, nullptr}, *y_ = nullptr, *tail_ = nullptr, *dt_ = nullptr, *decay_ = nullptr, *ssm_y_ = nullptr, *glu_ = nullptr, *logits_ = nullptr,
          *raw_ = nullptr;
    T *h_ = nullptr, *proj_ = nullptr, *xbc_ = nullptr, *act_ = nullptr, *hw_ = nullptr, *first_values_ = nullptr, *low_ = nullptr;
    float2 *table_ = nullptr;
    StepEntry *entries_ = nullptr;
    int *row_entry_ = nullptr, *tokens_ = nullptr, *want_ = nullptr, *history_ = nullptr;
    GenerateControl *gen_control_ = nullptr;
    size_t history_count_ = 0;
    void *host_ = nullptr;
    cudaGraphExec_t graph_ = nullptr;
    int graph_n_ = 0, graph_len_ = 0;
    int *graph_history_ = nullptr;
};

}  // namespace

// ---- C entry points (declared in include/gptb200.h) ------------------------------------------------------------------------

struct gptb200_decoder {
    std::unique_ptr<DecoderBase> model;
    gptb200_ctx *ctx;
};

namespace {

bool read_file(const std::string &path, std::string *out)
{
    FILE *f = fopen(path.c_str(), "rb");
    if (!f) return false;
    char buf[65536];
    size_t n;
    while ((n = fread(buf, 1, sizeof(buf), f)) > 0) out->append(buf, n);
    fclose(f);
    return true;
}

void keep_message(char *message, size_t capacity, const char *text)
{
    if (message && capacity > 0) snprintf(message, capacity, "%s", text);
}

}  // namespace

extern "C" {

int gptb200_decoder_check_config(const char *config_json, char *message, size_t capacity)
{
    if (!config_json) return GPTB200_ERR_INVALID_ARG;
    try {
        DecoderConfig::parse(config_json);
    } catch (const std::exception &e) {
        keep_message(message, capacity, e.what());
        return GPTB200_ERR_INVALID_ARG;
    }
    keep_message(message, capacity, "");
    return GPTB200_OK;
}

int gptb200_rotary_frequencies(int dims, double base, const double *scaling4, double *freq, double *gain)
{
    if (dims <= 0 || dims % 2 || !(base > 1.0) || !freq || !gain) return GPTB200_ERR_INVALID_ARG;
    RotaryConfig r;
    r.dims = dims;
    r.base = base;
    if (scaling4) {
        r.scaled = true;
        r.factor = scaling4[0];
        r.original = scaling4[1];
        r.fast = scaling4[2];
        r.slow = scaling4[3];
    }
    const std::vector<double> f = rotary_frequencies(r, gain);
    for (size_t i = 0; i < f.size(); ++i) freq[i] = f[i];
    return GPTB200_OK;
}

int gptb200_decoder_load(gptb200_decoder **out, const char *folder, int dtype, int device, void *cuda_stream, char *message, size_t capacity)
{
    if (!out || !folder || (dtype != GPTB200_DTYPE_BF16 && dtype != GPTB200_DTYPE_F32)) return GPTB200_ERR_INVALID_ARG;
    *out = nullptr;
    keep_message(message, capacity, "");
    gptb200_ctx *ctx = nullptr;
    std::unique_ptr<DecoderBase> model;
    int rc = GPTB200_OK;
    try {
        std::string text;
        if (!read_file(std::string(folder) + "/config.json", &text)) throw std::runtime_error(std::string("cannot read ") + folder + "/config.json");
        const DecoderConfig config = DecoderConfig::parse(text);
        rc = gptb200_ctx_create(&ctx, device, cuda_stream, GPTB200_MODE_3XTF32);
        if (rc != GPTB200_OK) {
            keep_message(message, capacity, gptb200_status_string(rc));
            return rc;
        }
        ctx->decode_early_launch = 1;   // no kernel of a step writes weights
        if (dtype == GPTB200_DTYPE_F32)
            model.reset(new DecoderModel<float>(ctx, config));
        else
            model.reset(new DecoderModel<__nv_bfloat16>(ctx, config));
        const SafeTensors file(std::string(folder) + "/model.safetensors");
        rc = model->load(file);
        if (rc != GPTB200_OK) keep_message(message, capacity, gptb200_last_error(ctx));
    } catch (const std::exception &e) {
        keep_message(message, capacity, e.what());
        rc = GPTB200_ERR_INVALID_ARG;
    }
    if (rc != GPTB200_OK) {
        model.reset();
        if (ctx) gptb200_ctx_destroy(ctx);
        return rc;
    }
    *out = new gptb200_decoder{std::move(model), ctx};
    return GPTB200_OK;
}

int gptb200_decoder_destroy(gptb200_decoder *d)
{
    if (!d) return GPTB200_ERR_INVALID_ARG;
    d->model.reset();
    gptb200_ctx_destroy(d->ctx);
    delete d;
    return GPTB200_OK;
}

gptb200_ctx *gptb200_decoder_context(gptb200_decoder *d) { return d ? d->ctx : nullptr; }
int gptb200_decoder_vocab(gptb200_decoder *d) { return d ? d->model->config().vocab : -1; }

int gptb200_decoder_open(gptb200_decoder *d, int max_len, int *slot) { return d ? d->model->open(max_len, slot) : GPTB200_ERR_INVALID_ARG; }
int gptb200_decoder_close(gptb200_decoder *d, int slot) { return d ? d->model->close(slot) : GPTB200_ERR_INVALID_ARG; }
int gptb200_decoder_length(gptb200_decoder *d, int slot) { return d ? d->model->length(slot) : -1; }

int gptb200_decoder_set_option(gptb200_decoder *d, const char *key, int value)
{
    return d && key ? d->model->set_option(key, value) : GPTB200_ERR_INVALID_ARG;
}

int gptb200_decoder_step(gptb200_decoder *d, int n, const int *slots, const int *counts, const int *tokens, int n_want, const int *want, float *logits)
{
    if (!d || n <= 0 || !slots || !counts || !tokens || n_want < 0 || (n_want > 0 && (!want || !logits))) return GPTB200_ERR_INVALID_ARG;
    return d->model->step(n, slots, counts, tokens, n_want, want, logits);
}

int gptb200_decoder_generate(gptb200_decoder *d, int n, const int *slots, const int *first, int steps, float temperature, unsigned long long seed, int *out)
{
    if (!d || !slots || !first || !out || !(temperature >= 0.0f)) return GPTB200_ERR_INVALID_ARG;
    return d->model->generate(n, slots, first, steps, temperature, seed, out);
}

int gptb200_sample_rows(gptb200_ctx *ctx, int *tokens, const float *logits, int rows, int vocab, long long pitch, float temperature, unsigned long long seed,
                        unsigned long long draw)
{
    if (!ctx || rows < 0 || vocab <= 0 || pitch < vocab || !(temperature >= 0.0f) || (rows > 0 && (!tokens || !logits))) return GPTB200_ERR_INVALID_ARG;
    if (rows == 0) return GPTB200_OK;
    sample_rows_kernel<<<rows, 512, 0, ctx->stream>>>(tokens, logits, vocab, pitch, temperature, seed, draw);
    ctx->launches++;
    CUDA_TRY(ctx, cudaGetLastError());
    return GPTB200_OK;
}

}  // extern "C"
