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

// ---- Zozonex: gated delta rule and windowed attention layers, output norms, squared-ReLU feed-forwards ----------
int32_t zozonex_parse(const JsonValue& root, Config& c) {
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
    c.embed_positions = true;
    const JsonValue* layers = root.find("layers");
    if (!layers || layers->kind != JsonValue::Array || layers->arr.empty()) return fail(LUMI_E_CONFIG, "config.json: 'layers' must be a non-empty array");
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
            LUMI_TRY(need_count(*mlp, "ff", where, 1, L.ff));
        }
        c.specs.push_back(L);
    }
    c.n_layers = (int)c.specs.size();
    return LUMI_OK;
}

int zozonex_shape(const Config& c, const std::string& name, int64_t shp[2], bool& wide) {
    wide = false;
    auto vec = [&](int64_t n) { shp[0] = n; return 1; };
    auto mat = [&](int64_t r, int64_t k) { shp[0] = r; shp[1] = k; return 2; };
    if (name == "embed") return mat(c.vocab, c.d_model);
    if (name == "final.norm") return vec(c.d_model);
    if (name.empty() || name[0] != 'l') return 0;
    const size_t dot = name.find('.');
    if (dot == std::string::npos || dot < 2 || dot > 9) return 0;
    int layer = 0;
    for (size_t i = 1; i < dot; ++i) {
        if (name[i] < '0' || name[i] > '9') return 0;
        layer = layer * 10 + (name[i] - '0');
    }
    if (layer >= c.n_layers) return 0;
    const LayerSpec& L = c.specs[layer];
    const MixerSpec& m = L.mixer;
    const std::string k = name.substr(dot + 1);
    const int64_t q = (int64_t)(m.kind == MIXER_DELTA ? m.kv_heads : m.heads) * m.dim, kk = (int64_t)m.kv_heads * m.dim;
    const int64_t v = (int64_t)(m.kind == MIXER_DELTA ? m.heads : m.kv_heads) * m.vdim, o = (int64_t)m.heads * m.vdim;
    if (k == "norm1") return vec(c.d_model);
    if (L.ff > 0) {
        if (k == "norm2") return vec(c.d_model);
        if (k == "mlp.up") return mat(L.ff, c.d_model);
        if (k == "mlp.down") return mat(c.d_model, L.ff);
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

const Architecture kArchitectures[] = {
    {"Zozonex", "", zozonex_parse, zozonex_shape},
};

}  // namespace

const Architecture* find_architecture(const char* name) {
    for (const Architecture& a : kArchitectures) if (strcmp(a.name, name) == 0) return &a;
    return nullptr;
}

}  // namespace lumi
