// Registry of the model designs whose config.json names one under "architecture", and their readers.  A config without
// that key is the Mamba-3 / attention hybrid (parse_config in api.cu).
#include "internal.h"
#include "json_min.h"

#include <cstring>

namespace lumi {
namespace {

int32_t need_number(const JsonValue& obj, const char* key, const std::string& where, double& out) {
    const JsonValue* v = obj.kind == JsonValue::Object ? obj.find(key) : nullptr;
    if (!v || v->kind != JsonValue::Number) return fail(LUMI_E_CONFIG, "config.json: %s needs a number '%s'", where.c_str(), key);
    out = v->num;
    return LUMI_OK;
}
int32_t need_count(const JsonValue& obj, const char* key, const std::string& where, int lowest, int& out) {
    double d = 0;
    LUMI_TRY(need_number(obj, key, where, d));
    if (d != (double)(int)d || d < lowest) return fail(LUMI_E_CONFIG, "config.json: %s: '%s' must be an integer >= %d", where.c_str(), key, lowest);
    out = (int)d;
    return LUMI_OK;
}
const JsonValue* object_at(const JsonValue& obj, const char* key) {
    const JsonValue* v = obj.kind == JsonValue::Object ? obj.find(key) : nullptr;
    return v && v->kind == JsonValue::Object ? v : nullptr;
}

// What the designs with a list of layers have in common at the top of their config.json.
int32_t parse_model_head(const JsonValue& root, Config& c, const JsonValue** layers) {
    LUMI_TRY(need_count(root, "vocab", "the model", 1, c.vocab));
    LUMI_TRY(need_count(root, "width", "the model", 1, c.d_model));
    double d = 0;
    const JsonValue* norm = object_at(root, "norm");
    const JsonValue* emb = object_at(root, "embedding");
    if (!norm || !emb) return fail(LUMI_E_CONFIG, "config.json: 'norm' and 'embedding' must be objects");
    LUMI_TRY(need_number(*norm, "eps", "norm", d));
    c.eps = (float)d;
    LUMI_TRY(need_number(*emb, "scale", "embedding", d));
    c.embed_scale = (float)d;
    *layers = root.find("layers");
    if (!*layers || (*layers)->kind != JsonValue::Array || (*layers)->arr.empty()) return fail(LUMI_E_CONFIG, "config.json: 'layers' must be a non-empty array");
    return LUMI_OK;
}

// ---- Zozonex: gated delta rule and windowed attention layers, output norms, squared-ReLU feed-forwards ----------
int32_t zozonex_parse(const JsonValue& root, Config& c) {
    const JsonValue* layers = nullptr;
    LUMI_TRY(parse_model_head(root, c, &layers));
    c.embed_positions = true;
    double d = 0;
    for (size_t i = 0; i < layers->arr.size(); ++i) {
        const JsonValue& e = layers->arr[i];
        const std::string where = "layer " + std::to_string(i);
        const JsonValue* type = e.kind == JsonValue::Object ? e.find("type") : nullptr;
        const JsonValue* mx = object_at(e, "mixer");
        if (!type || type->kind != JsonValue::String || !mx) return fail(LUMI_E_CONFIG, "config.json: %s needs a 'type' and a 'mixer'", where.c_str());
        LayerSpec L;
        MixerSpec& m = L.mixer;
        LUMI_TRY(need_count(*mx, "heads", where, 1, m.heads));
        LUMI_TRY(need_count(*mx, "kv_heads", where, 1, m.kv_heads));
        LUMI_TRY(need_count(*mx, "dim", where, 1, m.dim));
        LUMI_TRY(need_count(*mx, "vdim", where, 1, m.vdim));
        if (m.heads % m.kv_heads) return fail(LUMI_E_CONFIG, "config.json: %s: heads (%d) not divisible by kv_heads (%d)", where.c_str(), m.heads, m.kv_heads);
        if (type->str == "delta") {
            m.kind = MIXER_DELTA;
            LUMI_TRY(need_count(*mx, "conv", where, 1, m.taps));
        } else if (type->str == "attention") {
            m.kind = MIXER_ATTENTION;
            m.qk_norm = true;
            m.sink = true;
            m.sink_score = 0.f;
            LUMI_TRY(need_number(*mx, "scale", where, d));
            m.scale = (float)d;
            if (const JsonValue* mask = object_at(*mx, "mask")) LUMI_TRY(need_count(*mask, "size", where, 1, m.window));
            const JsonValue* from = mx->find("kv_from");
            if (from && from->kind != JsonValue::Null) {
                LUMI_TRY(need_count(*mx, "kv_from", where, 0, m.kv_from));
                if (m.kv_from >= (int)i) return fail(LUMI_E_CONFIG, "config.json: %s: kv_from must name an earlier layer", where.c_str());
                const MixerSpec& src = c.specs[m.kv_from].mixer;
                if (src.kind != MIXER_ATTENTION || src.kv_from >= 0)
                    return fail(LUMI_E_CONFIG, "config.json: %s: layer %d has no keys and values of its own", where.c_str(), m.kv_from);
                if (src.heads != m.heads || src.kv_heads != m.kv_heads || src.dim != m.dim || src.vdim != m.vdim)
                    return fail(LUMI_E_CONFIG, "config.json: %s: head sizes differ from those of layer %d", where.c_str(), m.kv_from);
            }
        } else {
            return fail(LUMI_E_CONFIG, "config.json: %s: mixer type '%s' is not known", where.c_str(), type->str.c_str());
        }
        const JsonValue* mlp = e.find("mlp");
        if (mlp && mlp->kind == JsonValue::Object) {
            const JsonValue* kind = mlp->find("kind");
            if (!kind || kind->kind != JsonValue::String || kind->str != "dense")
                return fail(LUMI_E_CONFIG, "config.json: %s: feed-forward kind '%s' is not known", where.c_str(), kind && kind->kind == JsonValue::String ? kind->str.c_str() : "?");
            LUMI_TRY(need_count(*mlp, "ff", where, 1, L.ff.ff));
        }
        c.specs.push_back(L);
    }
    c.n_layers = (int)c.specs.size();
    return LUMI_OK;
}

// "l<i>.<rest>": the layer's index, and the rest of the name; -1 for other names
int layer_of(const Config& c, const std::string& name, std::string& rest) {
    if (name.empty() || name[0] != 'l') return -1;
    const size_t dot = name.find('.');
    if (dot == std::string::npos || dot < 2 || dot > 9) return -1;
    int layer = 0;
    for (size_t i = 1; i < dot; ++i) {
        if (name[i] < '0' || name[i] > '9') return -1;
        layer = layer * 10 + (name[i] - '0');
    }
    if (layer >= c.n_layers) return -1;
    rest = name.substr(dot + 1);
    return layer;
}

int zozonex_shape(const Config& c, const std::string& name, int64_t shp[3], bool& wide) {
    wide = false;
    auto vec = [&](int64_t n) { shp[0] = n; return 1; };
    auto mat = [&](int64_t r, int64_t k) { shp[0] = r; shp[1] = k; return 2; };
    if (name == "embed") return mat(c.vocab, c.d_model);
    if (name == "final.norm") return vec(c.d_model);
    std::string k;
    const int layer = layer_of(c, name, k);
    if (layer < 0) return 0;
    const LayerSpec& L = c.specs[layer];
    const MixerSpec& m = L.mixer;
    const int64_t q = (int64_t)(m.kind == MIXER_DELTA ? m.kv_heads : m.heads) * m.dim, kk = (int64_t)m.kv_heads * m.dim;
    const int64_t v = (int64_t)(m.kind == MIXER_DELTA ? m.heads : m.kv_heads) * m.vdim, o = (int64_t)m.heads * m.vdim;
    if (k == "norm1") return vec(c.d_model);
    if (L.ff.ff > 0) {
        if (k == "norm2") return vec(c.d_model);
        if (k == "mlp.up") return mat(L.ff.ff, c.d_model);
        if (k == "mlp.down") return mat(c.d_model, L.ff.ff);
    }
    if (k == "mix.q") return mat(q, c.d_model);
    if (k == "mix.o") return mat(c.d_model, o);
    if (m.kv_from < 0) {
        if (k == "mix.k") return mat(kk, c.d_model);
        if (k == "mix.v") return mat(v, c.d_model);
    }
    if (m.kind == MIXER_DELTA) {
        wide = true;
        if (k == "mix.q.conv") return mat(q, m.taps);
        if (k == "mix.k.conv") return mat(kk, m.taps);
        if (k == "mix.v.conv") return mat(v, m.taps);
        wide = false;
        if (k == "mix.b" || k == "mix.a") return mat(m.heads, c.d_model);
        if (k == "mix.g") return mat(o, c.d_model);
        if (k == "mix.A_log" || k == "mix.dt_bias") return vec(m.heads);
        if (k == "mix.norm") return vec(m.vdim);
    }
    return 0;
}

// ---- Zutazen: retention, gated linear recurrence and latent attention layers behind norms of the stream, gated feed-forwards
// (dense with biases, or experts), a head of its own; layers may use another layer's weights --------------------------
int32_t zutazen_mixer(const JsonValue& mx, const std::string& type, const std::string& where, LayerSpec& L) {
    MixerSpec& m = L.mixer;
    double d = 0;
    auto rotation = [&](bool pairs) -> int32_t {
        const JsonValue* rot = object_at(mx, "rot");
        if (!rot) return fail(LUMI_E_CONFIG, "config.json: %s needs an object 'rot'", where.c_str());
        LUMI_TRY(need_count(*rot, "dims", where, 0, m.rot.dims));
        LUMI_TRY(need_number(*rot, "base", where, m.rot.base));
        if (m.rot.dims % 2 || m.rot.base <= 0) return fail(LUMI_E_CONFIG, "config.json: %s: rot.dims must be even and rot.base positive", where.c_str());
        m.rot.pairs = pairs;
        return LUMI_OK;
    };
    if (type == "retention") {
        m.kind = MIXER_RETENTION;
        LUMI_TRY(need_count(mx, "heads", where, 1, m.heads));
        LUMI_TRY(need_count(mx, "dim", where, 1, m.dim));
        LUMI_TRY(need_count(mx, "vdim", where, 1, m.vdim));
        m.kv_heads = m.heads;
        LUMI_TRY(rotation(false));
        if (m.rot.dims > m.dim) return fail(LUMI_E_CONFIG, "config.json: %s: rot.dims exceeds dim", where.c_str());
        const JsonValue* dec = mx.find("decay");
        if (!dec || dec->kind != JsonValue::Array || (int)dec->arr.size() != m.heads) return fail(LUMI_E_CONFIG, "config.json: %s: 'decay' must list one number per head", where.c_str());
        for (const JsonValue& v : dec->arr) {
            if (v.kind != JsonValue::Number || v.num < 0 || v.num > 1) return fail(LUMI_E_CONFIG, "config.json: %s: decays lie in [0, 1]", where.c_str());
            L.decay.push_back((float)v.num);
        }
        return LUMI_OK;
    }
    if (type == "rglru") {
        m.kind = MIXER_RGLRU;
        LUMI_TRY(need_count(mx, "width", where, 1, m.channels));
        LUMI_TRY(need_count(mx, "blocks", where, 1, m.blocks));
        LUMI_TRY(need_count(mx, "conv", where, 1, m.taps));
        if (m.channels % m.blocks) return fail(LUMI_E_CONFIG, "config.json: %s: width (%d) not divisible by blocks (%d)", where.c_str(), m.channels, m.blocks);
        return LUMI_OK;
    }
    if (type == "latent_attention") {
        m.kind = MIXER_LATENT;
        LUMI_TRY(need_count(mx, "heads", where, 1, m.heads));
        LUMI_TRY(need_count(mx, "dim", where, 1, m.dim));
        LUMI_TRY(need_count(mx, "rot_dim", where, 0, m.rot_dim));
        LUMI_TRY(need_count(mx, "vdim", where, 1, m.vdim));
        LUMI_TRY(need_count(mx, "kv_rank", where, 1, m.kv_rank));
        m.kv_heads = m.heads;
        LUMI_TRY(need_number(mx, "scale", where, d));
        m.scale = (float)d;
        LUMI_TRY(rotation(true));
        if (m.rot.dims != m.rot_dim) return fail(LUMI_E_CONFIG, "config.json: %s: rot.dims must equal rot_dim", where.c_str());
        if (const JsonValue* mask = object_at(mx, "mask")) LUMI_TRY(need_count(*mask, "size", where, 1, m.window));
        return LUMI_OK;
    }
    return fail(LUMI_E_CONFIG, "config.json: %s: mixer type '%s' is not known", where.c_str(), type.c_str());
}

int32_t zutazen_parse(const JsonValue& root, Config& c) {
    const JsonValue* layers = nullptr;
    LUMI_TRY(parse_model_head(root, c, &layers));
    c.own_head = true;
    c.norm_offset = false;
    for (size_t i = 0; i < layers->arr.size(); ++i) {
        const JsonValue& e = layers->arr[i];
        const std::string where = "layer " + std::to_string(i);
        const JsonValue* type = e.kind == JsonValue::Object ? e.find("type") : nullptr;
        const JsonValue* mx = object_at(e, "mixer");
        if (!type || type->kind != JsonValue::String || !mx) return fail(LUMI_E_CONFIG, "config.json: %s needs a 'type' and a 'mixer'", where.c_str());
        LayerSpec L;
        L.pre_norm = true;
        LUMI_TRY(zutazen_mixer(*mx, type->str, where, L));
        if (const JsonValue* mlp = object_at(e, "mlp")) {
            const JsonValue* kind = mlp->find("kind");
            const std::string k = kind && kind->kind == JsonValue::String ? kind->str : "?";
            if (k == "dense") {
                L.ff.act = ACT_RELU_GATE;
                L.ff.bias = true;
                LUMI_TRY(need_count(*mlp, "ff", where, 1, L.ff.ff));
            } else if (k == "moe") {
                const JsonValue* ex = object_at(*mlp, "expert");
                const JsonValue* ro = object_at(*mlp, "router");
                if (!ex || !ro) return fail(LUMI_E_CONFIG, "config.json: %s: 'expert' and 'router' must be objects", where.c_str());
                L.ff.act = ACT_SILU_GATE;
                LUMI_TRY(need_count(*ex, "ff", where, 1, L.ff.ff));
                LUMI_TRY(need_count(*ro, "experts", where, 1, L.ff.experts));
                LUMI_TRY(need_count(*ro, "top", where, 1, L.ff.top));
                if (L.ff.top > L.ff.experts) return fail(LUMI_E_CONFIG, "config.json: %s: router.top exceeds router.experts", where.c_str());
            } else {
                return fail(LUMI_E_CONFIG, "config.json: %s: feed-forward kind '%s' is not known", where.c_str(), k.c_str());
            }
        }
        const JsonValue* from = e.find("weights_of");
        if (from && from->kind != JsonValue::Null) {
            LUMI_TRY(need_count(e, "weights_of", where, 0, L.weights_of));
            if (L.weights_of >= (int)i) return fail(LUMI_E_CONFIG, "config.json: %s: weights_of must name an earlier layer", where.c_str());
            while (c.specs[L.weights_of].weights_of >= 0) L.weights_of = c.specs[L.weights_of].weights_of;
            const LayerSpec& S = c.specs[L.weights_of];
            if (S.mixer.kind != L.mixer.kind || S.mixer.heads != L.mixer.heads || S.mixer.dim != L.mixer.dim || S.mixer.vdim != L.mixer.vdim ||
                S.mixer.kv_rank != L.mixer.kv_rank || S.mixer.rot_dim != L.mixer.rot_dim || S.mixer.channels != L.mixer.channels ||
                S.mixer.blocks != L.mixer.blocks || S.mixer.taps != L.mixer.taps || S.ff.ff != L.ff.ff || S.ff.act != L.ff.act || S.ff.experts != L.ff.experts)
                return fail(LUMI_E_CONFIG, "config.json: %s: sizes differ from those of layer %d", where.c_str(), L.weights_of);
        }
        c.specs.push_back(L);
    }
    c.n_layers = (int)c.specs.size();
    return LUMI_OK;
}

int zutazen_shape(const Config& c, const std::string& name, int64_t shp[3], bool& wide) {
    wide = false;
    auto vec = [&](int64_t n) { shp[0] = n; return 1; };
    auto mat = [&](int64_t r, int64_t k) { shp[0] = r; shp[1] = k; return 2; };
    auto fp32 = [&](int rank) { wide = true; return rank; };
    if (name == "embed" || name == "head") return mat(c.vocab, c.d_model);
    if (name == "final.norm") return vec(c.d_model);
    std::string k;
    const int layer = layer_of(c, name, k);
    if (layer < 0 || c.specs[layer].weights_of >= 0) return 0;
    const LayerSpec& L = c.specs[layer];
    const MixerSpec& m = L.mixer;
    const int64_t D = c.d_model, H = m.heads;
    if (k == "norm1") return vec(D);
    if (L.ff.ff > 0) {
        if (k == "norm2") return vec(D);
        if (L.ff.experts == 0) {
            if (k == "mlp.gate" || k == "mlp.up") return mat(L.ff.ff, D);
            if (k == "mlp.down") return mat(D, L.ff.ff);
            if (k == "mlp.gate.b" || k == "mlp.up.b") return vec(L.ff.ff);
            if (k == "mlp.down.b") return vec(D);
        } else {
            if (k == "mlp.router") return mat(L.ff.experts, D);
            if (k.rfind("mlp.e", 0) == 0) {
                const size_t dot = k.find('.', 5);
                if (dot == std::string::npos || dot == 5 || dot > 12) return 0;
                int e = 0;
                for (size_t i = 5; i < dot; ++i) {
                    if (k[i] < '0' || k[i] > '9') return 0;
                    e = e * 10 + (k[i] - '0');
                }
                if (e >= L.ff.experts) return 0;
                const std::string part = k.substr(dot + 1);
                if (part == "gate" || part == "up") return mat(L.ff.ff, D);
                if (part == "down") return mat(D, L.ff.ff);
                return 0;
            }
        }
    }
    if (m.kind == MIXER_RETENTION) {
        if (k == "mix.q" || k == "mix.k") return mat(H * m.dim, D);
        if (k == "mix.v" || k == "mix.g") return mat(H * m.vdim, D);
        if (k == "mix.o") return mat(D, H * m.vdim);
    } else if (m.kind == MIXER_RGLRU) {
        const int64_t C = m.channels, bs = m.channels / m.blocks;
        if (k == "mix.y" || k == "mix.x") return mat(C, D);
        if (k == "mix.y.b" || k == "mix.x.b" || k == "mix.conv.b" || k == "mix.lam") return vec(C);
        if (k == "mix.conv") { mat(C, m.taps); return fp32(2); }
        if (k == "mix.ra" || k == "mix.ri") { shp[0] = m.blocks; shp[1] = shp[2] = bs; return 3; }
        if (k == "mix.ra.b" || k == "mix.ri.b") { mat(m.blocks, bs); return fp32(2); }
        if (k == "mix.o") return mat(D, C);
    } else if (m.kind == MIXER_LATENT) {
        if (k == "mix.q") return mat(H * (m.dim + m.rot_dim), D);
        if (k == "mix.dkv") return mat(m.kv_rank + m.rot_dim, D);
        if (k == "mix.dkv.norm") return vec(m.kv_rank);
        if (k == "mix.uk") return mat(H * m.dim, m.kv_rank);
        if (k == "mix.uv") return mat(H * m.vdim, m.kv_rank);
        if (k == "mix.g") return mat(H * m.vdim, D);
        if (k == "mix.o") return mat(D, H * m.vdim);
    }
    return 0;
}

const Architecture kArchitectures[] = {
    {"Zozonex", "", zozonex_parse, zozonex_shape},
    {"Zutazen", "", zutazen_parse, zutazen_shape},
};

}  // namespace

const Architecture* find_architecture(const char* name) {
    for (const Architecture& a : kArchitectures) if (strcmp(a.name, name) == 0) return &a;
    return nullptr;
}

}  // namespace lumi
