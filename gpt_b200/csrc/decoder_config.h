// Configuration of the decoder models that are described by a config.json (host only): the architectures the library knows, what
// each of them fixes, and the sizes and constants that a model's file gives.
#pragma once

#include <algorithm>
#include <cmath>

#include "json_lite.h"

namespace gptb200 {

// Rotary positions: pairs (i, i + dims / 2), frequency base^(-2 i / dims), optionally stretched (YaRN).
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

enum class MixerKind { Mamba2, Latent };

struct LayerConfig {
    MixerKind kind;
    Mamba2Config mamba{};
    LatentConfig latent{};
    int ff = 0;   // width of the gated feed-forward, 0: none
};

// What an architecture fixes.  All of them: layer norms with bias before and after each sublayer, gated GELU feed-forwards.
struct ArchitectureTraits {
    const char *name;
    bool token_shift;     // the mixer input is blended with the previous token's
    bool depth_average;   // weighted sum over the results of all earlier layers after each layer
    bool token_side;      // gated per-layer token embedding after the feed-forward
};

inline const std::vector<ArchitectureTraits> &known_architectures()
{
    static const std::vector<ArchitectureTraits> known = {{"Budurax", true, true, true}};
    return known;
}

struct DecoderConfig {
    ArchitectureTraits traits{};
    int vocab = 0, width = 0, side_dim = 0;
    double eps = 0.0;
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
        const Json &layers = j.at("layers");
        if (layers.kind != Json::Array || layers.items.empty()) throw std::runtime_error("'layers' is not a list of layers");
        for (size_t i = 0; i < layers.items.size(); ++i) {
            try {
                c.layers.push_back(parse_layer(layers.items[i], static_cast<int>(i), c.layers));
            } catch (const std::exception &e) {
                throw std::runtime_error("layer " + std::to_string(i) + ": " + e.what());
            }
        }
        return c;
    }

private:
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
    static LayerConfig parse_layer(const Json &j, int index, const std::vector<LayerConfig> &before)
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
