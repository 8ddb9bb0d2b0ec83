// Registry of model designs.  See model_spec.h.
#include "model_spec.h"

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstring>

namespace hm {
namespace {

bool fail(std::string* err, const std::string& m) {
    *err = "config.json: " + m;
    return false;
}

// A positive integer, or nothing.
bool get_int(const Json& o, const char* key, int* out) {
    const Json* v = o.get(key);
    if (!v || v->kind != Json::Num || v->num < 1 || v->num > 2147483647.0 || v->num != std::floor(v->num)) return false;
    *out = (int)v->num;
    return true;
}
bool is_null(const Json* v) { return !v || v->kind == Json::Null; }

// Tunitar: latent attention without positions, squared-ReLU MLPs (or none), grouped norms, token shift, layer scales.
bool read_tunitar(const Json& j, ModelSpec* s, std::string* err) {
    hm_config& c = s->cfg;
    s->token_shift = s->layer_scale = true;
    if (!get_int(j, "width", &c.hidden_size) || !get_int(j, "vocab", &c.vocab_size)) return fail(err, "missing `width` or `vocab`");
    const Json* norm = j.get("norm");
    const Json* eps = norm ? norm->get("eps") : nullptr;
    if (!norm || !get_int(*norm, "groups", &s->norm_groups) || !eps || eps->kind != Json::Num) return fail(err, "`norm` needs `groups` and `eps`");
    if (c.hidden_size % s->norm_groups != 0) return fail(err, "`norm.groups` does not divide `width`");
    c.rms_norm_eps = eps->num;
    const Json* list = j.get("layers");
    if (!list || list->kind != Json::Arr || list->arr.empty()) return fail(err, "missing `layers`");
    for (size_t i = 0; i < list->arr.size(); ++i) {
        const Json& e = list->arr[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        LayerSpec l;
        const Json* type = e.get("type");
        if (!type || type->kind != Json::Str || type->str != "latent_attention") return fail(err, at + "unknown mixer type");
        l.mixer = MIX_LATENT;
        const Json* m = e.get("mixer");
        const Json* scale = m ? m->get("scale") : nullptr;
        if (!m || !get_int(*m, "heads", &l.heads) || !get_int(*m, "dim", &l.dim) || !get_int(*m, "vdim", &l.vdim) || !get_int(*m, "kv_rank", &l.kv_rank) || !scale || scale->kind != Json::Num)
            return fail(err, at + "the mixer needs heads, dim, vdim, kv_rank and scale");
        l.scale = (float)scale->num;
        const Json* from = m->get("kv_from");
        if (!is_null(from)) {
            if (from->kind != Json::Num || from->num < 0 || from->num != std::floor(from->num) || from->num >= (double)i) return fail(err, at + "`kv_from` must name an earlier layer");
            l.kv_from = (int)from->num;
            const LayerSpec& o = s->layers[l.kv_from];
            if (o.kv_from >= 0) return fail(err, at + "`kv_from` names a layer without latents of its own");
            if (o.kv_rank != l.kv_rank) return fail(err, at + "`kv_from` names a layer of another kv_rank");
        }
        const Json* mlp = e.get("mlp");
        if (!is_null(mlp)) {
            const Json* kind = mlp->get("kind");
            if (!kind || kind->kind != Json::Str || kind->str != "dense" || !get_int(*mlp, "ff", &l.ff)) return fail(err, at + "unknown mlp");
            l.mlp = MLP_SQRELU;
        }
        c.num_attention_heads = std::max(c.num_attention_heads, l.heads);
        c.head_dim = std::max(c.head_dim, l.dim);
        c.intermediate_size = std::max(c.intermediate_size, l.ff);
        s->layers.push_back(l);
    }
    c.num_hidden_layers = (int)s->layers.size();
    c.num_key_value_heads = 1;
    c.max_position_embeddings = 1 << 30;  // no positions: the cache is the only limit
    c.intermediate_size = std::max(c.intermediate_size, 1);
    return true;
}

struct Design {
    const char* name;
    bool (*read)(const Json&, ModelSpec*, std::string*);
};
const Design kDesigns[] = {{"Tunitar", read_tunitar}};

}  // namespace

bool parse_model_spec(const char* text, size_t len, ModelSpec* out, std::string* err) {
    Json j;
    if (!json_parse(text, len, &j, err)) return false;
    if (j.kind != Json::Obj) return fail(err, "top level is not an object");
    *out = ModelSpec();
    const Json* arch = j.get("architecture");
    if (arch && arch->kind == Json::Str) {
        for (const Design& d : kDesigns)
            if (arch->str == d.name) {
                out->arch = d.name;
                if (!d.read(j, out, err)) return false;
                auto tok = [&](const char* k) {
                    const Json* v = j.get(k);
                    return v && v->kind == Json::Num ? (uint32_t)v->num : UINT32_MAX;
                };
                out->cfg.eos_token_id = tok("eos_token_id");
                out->cfg.bos_token_id = tok("bos_token_id");
                return true;
            }
        return fail(err, "unknown architecture `" + arch->str + "`");
    }
    return config_from_json(j, &out->cfg, err);
}

bool parse_model_spec_file(const std::string& path, ModelSpec* out, std::string* err) {
    MappedFile f;
    if (!f.open(path, err)) return false;
    return parse_model_spec(reinterpret_cast<const char*>(f.data()), f.size(), out, err);
}

std::string layers_json(const ModelSpec& spec) {
    std::string o = "[";
    for (size_t i = 0; i < spec.layers.size(); ++i) {
        const LayerSpec& l = spec.layers[i];
        char t[320];
        std::snprintf(t, sizeof(t), "%s{\"type\":\"latent_attention\",\"heads\":%d,\"dim\":%d,\"vdim\":%d,\"kv_rank\":%d,\"kv_from\":%s,\"scale\":%.9g,\"ff\":%d}", i ? "," : "", l.heads, l.dim, l.vdim, l.kv_rank,
                      l.kv_from < 0 ? "null" : std::to_string(l.kv_from).c_str(), l.scale, l.ff);
        o += t;
    }
    return o + "]";
}

}  // namespace hm
