// Configuration of the decoder models that are described by a config.json (host only): the architectures the library knows, what
// each of them fixes, and the sizes and constants that a model's file gives.
#pragma once

#include <algorithm>
#include <cmath>

#include "json_lite.h"

namespace gptb200 {

// Rotary positions: frequency base^(-2 i / dims) of pair i, optionally stretched (YaRN).  Which dimensions form a pair -- (i, i + dims / 2)
// or (2 i, 2 i + 1) -- is fixed by the layer kind.
struct RotaryConfig {
    int dims = 0;
    double base = 0.0;
    bool scaled = false;
    double factor = 1.0, original = 0.0, fast = 0.0, slow = 0.0;
    bool operator==(const RotaryConfig &o) const
    {
        return dims == o.dims && base == o.base && scaled == o.scaled && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow;
    }
};

// Frequencies of the dims / 2 pairs and the factor on cosine and sine.
inline std::vector<double> rotary_frequencies(const RotaryConfig &r, double *gain)
{
    const double pi = 3.14159265358979323846;
    std::vector<double> f(r.dims / 2);
    for (int i = 0; i < r.dims / 2; ++i) f[i] = std::pow(r.base, -2.0 * i / r.dims);
    *gain = 1.0;
    if (!r.scaled) return f;
    // dimension whose wave makes `turns` turns over the original length
    const auto dimension = [&](double turns) { return r.dims * std::log(r.original / (2.0 * pi * turns)) / (2.0 * std::log(r.base)); };
    const double lo = std::max(std::floor(dimension(r.fast)), 0.0), hi = std::min(std::ceil(dimension(r.slow)), r.dims - 1.0);
    for (int i = 0; i < r.dims / 2; ++i) {
        const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
        f[i] = f[i] / r.factor * ramp + f[i] * (1.0 - ramp);
    }
    *gain = 0.1 * std::log(r.factor) + 1.0;
    return f;
}

struct Mamba2Config {
    int heads, vdim, state, groups, conv, norm_groups;
    int inner() const { return heads * vdim; }
    int conv_channels() const { return inner() + 2 * groups * state; }
};

struct LatentConfig {
    int heads, dim, rot_dim, vdim, kv_rank;
    int kv_from = -1;   // layer whose latent and rotated key part this layer attends to
    double scale;
    RotaryConfig rot;
};

// Softmax attention with grouped key / value heads, biased projections, rotated neighbouring dimensions and a sigmoid output gate.
struct GroupedConfig {
    int heads, kv_heads, dim, vdim;
    double scale;
    double softcap = 0.0;   // scores become softcap * tanh(score / softcap); 0: they stay
    bool value_mix = false; // values are blended with those of the first layer that says so
    bool first_values = false;   // this is that layer
    RotaryConfig rot;
};

// Linear attention with one constant decay per head (S <- decay S + k v^T, read after the update).
struct LightningConfig {
    int heads, dim, vdim;
    std::vector<double> decay;
};

// Linear attention with a decay per key channel and token and a bonus for the current token (read before the update).
struct WkvConfig {
    int heads, dim;
};

enum class MixerKind { Mamba2, Latent, Grouped, Lightning, Wkv };

struct LayerConfig {
    MixerKind kind;
    Mamba2Config mamba{};
    LatentConfig latent{};
    GroupedConfig grouped{};
    LightningConfig lightning{};
    WkvConfig wkv{};
    int ff = 0;   // width of the gated feed-forward, 0: none
};

// How the residual stream is normed around the sublayers.
enum class NormScheme {
    LayerNormAround,   // layer norms with bias before and after each sublayer: x += norm(sublayer(norm(x)))
    RmsBefore,         // root-mean-square norm, weight stored as its distance from one: x += residual_mult * sublayer(norm(x))
};

// What an architecture fixes.  All of them: gated feed-forwards.
struct ArchitectureTraits {
    const char *name;
    NormScheme norms;
    bool token_shift;     // the mixer input is blended with the previous token's
    bool depth_average;   // weighted sum over the results of all earlier layers after each layer
    bool token_side;      // gated per-layer token embedding after the feed-forward
    bool silu_gate;       // feed-forward gates: silu (GELU otherwise)
    bool pair_embedding;  // embedding times a constant, plus a row for the hashed pair (previous token, token)
};

inline const std::vector<ArchitectureTraits> &known_architectures()
{
    static const std::vector<ArchitectureTraits> known = {{"Budurax", NormScheme::LayerNormAround, true, true, true, false, false},
                                                          {"Lutelorn", NormScheme::RmsBefore, false, false, false, true, true}};
    return known;
}

struct DecoderConfig {
    ArchitectureTraits traits{};
    int vocab = 0, width = 0, side_dim = 0;
    double eps = 0.0;
    double residual_mult = 1.0, embed_scale = 1.0;
    long long pair_buckets = 0, pair_mul_previous = 0, pair_mul_current = 0;   // buckets 0: no pair embedding
    std::vector<LayerConfig> layers;

    static DecoderConfig parse(const std::string &text)
    {
        const Json j = Json::parse(text);
        DecoderConfig c;
        const std::string &name = j.str("architecture");
        bool known = false;
        for (const ArchitectureTraits &t : known_architectures())
            if (name == t.name) {
                c.traits = t;
                known = true;
            }
        if (!known) throw std::runtime_error("unknown architecture '" + name + "'");
        c.vocab = j.size("vocab");
        c.width = j.size("width");
        c.eps = j.at("norm").num("eps");
        if (c.traits.token_side) c.side_dim = j.at("token_side").size("dim");
        if (c.traits.norms == NormScheme::RmsBefore) c.residual_mult = j.num("residual_mult");
        if (c.traits.pair_embedding) {
            const Json &e = j.at("embedding");
            c.embed_scale = e.num("scale");
            if (e.has("bigram")) {
                const Json &b = e.at("bigram");
                c.pair_buckets = b.size("buckets");
                c.pair_mul_previous = multiplier(b, "mul_prev");
                c.pair_mul_current = multiplier(b, "mul_cur");
            }
        }
        const Json &layers = j.at("layers");
        if (layers.kind != Json::Array || layers.items.empty()) throw std::runtime_error("'layers' is not a list of layers");
        for (size_t i = 0; i < layers.items.size(); ++i) {
            try {
                c.layers.push_back(parse_layer(layers.items[i], static_cast<int>(i), c.layers, c.traits));
            } catch (const std::exception &e) {
                throw std::runtime_error("layer " + std::to_string(i) + ": " + e.what());
            }
        }
        return c;
    }

private:
    // products with token ids stay far below 2^63
    static long long multiplier(const Json &j, const char *key)
    {
        const double v = j.num(key);
        if (!(v >= 0.0 && v <= 2147483647.0) || v != std::floor(v)) throw std::runtime_error(std::string("'") + key + "' is not a non-negative integer");
        return static_cast<long long>(v);
    }
    static RotaryConfig parse_rotary(const Json &j)
    {
        RotaryConfig r;
        r.dims = j.size("dims");
        r.base = j.num("base");
        if (r.dims % 2 || !(r.base > 1.0)) throw std::runtime_error("rotary sizes");
        if (j.has("scaling")) {
            const Json &s = j.at("scaling");
            r.scaled = true;
            r.factor = s.num("factor");
            r.original = s.num("original");
            r.fast = s.num("fast");
            r.slow = s.num("slow");
            if (!(r.factor > 0.0 && r.original > 0.0 && r.fast > 0.0 && r.slow > 0.0)) throw std::runtime_error("rotary scaling");
        }
        return r;
    }
    static LayerConfig parse_layer(const Json &j, int index, const std::vector<LayerConfig> &before, const ArchitectureTraits &traits)
    {
        LayerConfig l{};
        const std::string &type = j.str("type");
        const Json &m = j.at("mixer");
        if (type == "mamba2") {
            l.kind = MixerKind::Mamba2;
            l.mamba = {m.size("heads"), m.size("vdim"), m.size("state"), m.size("groups"), m.size("conv"), m.size("norm_groups")};
            if (l.mamba.heads % l.mamba.groups) throw std::runtime_error("'heads' is not a multiple of 'groups'");
            if (l.mamba.inner() % l.mamba.norm_groups) throw std::runtime_error("heads * vdim is not a multiple of 'norm_groups'");
        } else if (type == "latent_attention") {
            l.kind = MixerKind::Latent;
            LatentConfig &a = l.latent;
            a.heads = m.size("heads");
            a.dim = m.size("dim");
            a.rot_dim = m.size("rot_dim");
            a.vdim = m.size("vdim");
            a.kv_rank = m.size("kv_rank");
            a.scale = m.num("scale");
            a.rot = parse_rotary(m.at("rot"));
            if (a.rot.dims > a.rot_dim) throw std::runtime_error("more rotated dimensions than 'rot_dim'");
            if (m.has("kv_from")) {
                const double f = m.num("kv_from");
                if (!(f >= 0 && f < index) || f != std::floor(f)) throw std::runtime_error("'kv_from' is not an earlier layer");
                a.kv_from = static_cast<int>(f);
                const LayerConfig &src = before[a.kv_from];
                if (src.kind != MixerKind::Latent || src.latent.kv_from >= 0) throw std::runtime_error("'kv_from' is not a layer with keys of its own");
                if (src.latent.kv_rank != a.kv_rank || src.latent.rot_dim != a.rot_dim || !(src.latent.rot == a.rot))
                    throw std::runtime_error("'kv_from': latent sizes or rotation differ");
            }
        } else if (type == "attention") {
            l.kind = MixerKind::Grouped;
            GroupedConfig &a = l.grouped;
            a.heads = m.size("heads");
            a.kv_heads = m.size("kv_heads");
            a.dim = m.size("dim");
            a.vdim = m.size("vdim");
            if (a.heads % a.kv_heads) throw std::runtime_error("'heads' is not a multiple of 'kv_heads'");
            a.scale = m.num("scale");
            if (m.has("softcap")) {
                a.softcap = m.num("softcap");
                if (!(a.softcap > 0.0)) throw std::runtime_error("'softcap' is not positive");
            }
            if (m.has("rot")) a.rot = parse_rotary(m.at("rot"));
            if (a.rot.dims > a.dim) throw std::runtime_error("more rotated dimensions than 'dim'");
            a.value_mix = m.has("v_mix") && m.flag("v_mix");
            if (a.value_mix) {
                a.first_values = true;
                for (const LayerConfig &b : before)
                    if (b.kind == MixerKind::Grouped && b.grouped.first_values) {
                        a.first_values = false;
                        if (b.grouped.kv_heads != a.kv_heads || b.grouped.vdim != a.vdim) throw std::runtime_error("'v_mix': the first such layer's values have other sizes");
                    }
            }
        } else if (type == "lightning") {
            l.kind = MixerKind::Lightning;
            LightningConfig &a = l.lightning;
            a.heads = m.size("heads");
            a.dim = m.size("dim");
            a.vdim = m.size("vdim");
            const Json &d = m.at("decay");
            if (d.kind != Json::Array || d.items.size() != static_cast<size_t>(a.heads)) throw std::runtime_error("'decay' is not a list with one number per head");
            for (const Json &v : d.items) {
                if (v.kind != Json::Number || !(v.number >= 0.0 && v.number <= 1.0)) throw std::runtime_error("'decay' is not between 0 and 1");
                a.decay.push_back(v.number);
            }
        } else if (type == "wkv") {
            l.kind = MixerKind::Wkv;
            l.wkv = {m.size("heads"), m.size("dim")};
            if (traits.norms != NormScheme::RmsBefore) throw std::runtime_error("'wkv' layers mix their own inputs: not with this architecture's norms");
        } else {
            throw std::runtime_error("unknown layer type '" + type + "'");
        }
        if (j.has("mlp")) {
            const Json &f = j.at("mlp");
            if (f.str("kind") != "dense") throw std::runtime_error("unknown feed-forward '" + f.str("kind") + "'");
            l.ff = f.size("ff");
        }
        return l;
    }
};

}  // namespace gptb200
