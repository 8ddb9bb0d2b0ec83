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
bool get_num(const Json& o, const char* key, double* out) {
    const Json* v = o.get(key);
    if (!v || v->kind != Json::Num) return false;
    *out = v->num;
    return true;
}
// A count that may be zero, absent or null.
bool get_count(const Json& o, const char* key, int* out) {
    const Json* v = o.get(key);
    *out = 0;
    if (is_null(v) || (v->kind == Json::Num && v->num == 0)) return true;
    return get_int(o, key, out);
}

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

// Grouped-query attention of the layer lists: query and key norms per head or over the whole projection, query temperature,
// distance bias, blended values.
bool read_gqa_mixer(const Json& m, bool positional, LayerSpec* l, const std::string& at, std::string* err) {
    double scale = 0;
    l->mixer = MIX_GQA;
    if (!get_int(m, "heads", &l->heads) || !get_int(m, "kv_heads", &l->kv_heads) || !get_int(m, "dim", &l->dim) || !get_int(m, "vdim", &l->vdim) || !get_num(m, "scale", &scale))
        return fail(err, at + "the mixer needs heads, kv_heads, dim, vdim and scale");
    if (l->heads % l->kv_heads != 0) return fail(err, at + "`kv_heads` does not divide `heads`");
    l->scale = (float)scale;
    l->qk_norm = positional ? QKN_ALL : QKN_HEAD;
    const Json* mix = m.get("v_mix");
    if (!is_null(mix) && mix->kind != Json::Bool) return fail(err, at + "`v_mix` must be true or false");
    l->v_mix = !is_null(mix) && mix->b;
    if (!positional) return true;
    if (!get_num(m, "bias_max", &l->bias_reach) || l->bias_reach <= 0 || l->bias_reach > 1 << 20) return fail(err, at + "`bias_max` must be a positive number of tokens");
    const Json* t = m.get("q_temp");
    if (!is_null(t)) {
        double coef = 0;
        if (!get_num(*t, "coef", &coef) || !get_int(*t, "every", &l->temp_every)) return fail(err, at + "`q_temp` needs coef and every");
        l->temp_coef = (float)coef;
    }
    return true;
}

bool read_moe(const Json& f, LayerSpec* l, const std::string& at, std::string* err) {
    const Json *kind = f.get("kind"), *ex = f.get("expert"), *r = f.get("router");
    double limit = 0;
    if (!kind || kind->kind != Json::Str || kind->str != "moe") return fail(err, at + "unknown mlp");
    if (!ex || !get_int(*ex, "ff", &l->ff) || !get_num(*ex, "limit", &limit)) return fail(err, at + "`mlp.expert` needs ff and limit");
    if (!r || !get_int(*r, "experts", &l->experts) || !get_int(*r, "top", &l->top) || !get_count(*r, "identity", &l->identity)) return fail(err, at + "`mlp.router` needs experts and top");
    if (l->top > l->experts + l->identity) return fail(err, at + "`mlp.router.top` is larger than the number of router outputs");
    l->limit = (float)limit;
    l->mlp = MLP_MOE;
    return true;
}

// Dipisun: grouped-query attention in two kinds, norms on what the sublayers give back, mixtures of experts (or none).
bool read_dipisun(const Json& j, ModelSpec* s, std::string* err) {
    hm_config& c = s->cfg;
    s->post_norm = s->sin_pos = true;
    if (!get_int(j, "width", &c.hidden_size) || !get_int(j, "vocab", &c.vocab_size)) return fail(err, "missing `width` or `vocab`");
    const Json* norm = j.get("norm");
    double mult = 0;
    if (!norm || !get_num(*norm, "eps", &c.rms_norm_eps)) return fail(err, "`norm` needs `eps`");
    if (!get_num(j, "residual_mult", &mult)) return fail(err, "missing `residual_mult`");
    s->residual_mult = (float)mult;
    const Json* list = j.get("layers");
    if (!list || list->kind != Json::Arr || list->arr.empty()) return fail(err, "missing `layers`");
    int first = -1;
    for (size_t i = 0; i < list->arr.size(); ++i) {
        const Json& e = list->arr[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        LayerSpec l;
        const Json *type = e.get("type"), *m = e.get("mixer"), *mlp = e.get("mlp");
        const bool positional = type && type->kind == Json::Str && type->str == "attention";
        if (!positional && !(type && type->kind == Json::Str && type->str == "attention_2")) return fail(err, at + "unknown mixer type");
        if (!m) return fail(err, at + "missing `mixer`");
        if (!read_gqa_mixer(*m, positional, &l, at, err)) return false;
        if (l.v_mix) {
            if (first < 0) first = (int)i;
            l.v_first = first;
            if (first < (int)i && s->layers[first].kv_heads * s->layers[first].vdim != l.kv_heads * l.vdim) return fail(err, at + "`v_mix` blends values of another size");
        }
        if (!is_null(mlp) && !read_moe(*mlp, &l, at, err)) return false;
        c.num_attention_heads = std::max(c.num_attention_heads, l.heads);
        c.num_key_value_heads = std::max(c.num_key_value_heads, l.kv_heads);
        c.head_dim = std::max(c.head_dim, l.dim);
        c.intermediate_size = std::max(c.intermediate_size, l.ff);
        s->layers.push_back(l);
    }
    c.num_hidden_layers = (int)s->layers.size();
    c.max_position_embeddings = 1 << 30;  // positions are computed: the cache is the only limit
    c.intermediate_size = std::max(c.intermediate_size, 1);
    return true;
}

bool get_str(const Json& o, const char* key, std::string* out) {
    const Json* v = o.get(key);
    if (!v || v->kind != Json::Str) return false;
    *out = v->str;
    return true;
}

bool read_rotation(const Json& m, int dim, RotSpec* r, const std::string& at, std::string* err) {
    const Json* j = m.get("rot");
    if (is_null(j)) return fail(err, at + "the mixer needs `rot`");
    if (!get_int(*j, "dims", &r->dims) || !get_num(*j, "base", &r->base) || r->base <= 0) return fail(err, at + "`rot` needs dims and base");
    if (r->dims % 2 != 0 || r->dims > dim) return fail(err, at + "`rot.dims` must be even and at most the head size");
    const Json* s = j->get("scaling");
    if (is_null(s)) return true;
    r->scaled = true;
    if (!get_num(*s, "factor", &r->factor) || !get_num(*s, "low", &r->low) || !get_num(*s, "high", &r->high) || !get_num(*s, "original", &r->original)) return fail(err, at + "`rot.scaling` needs factor, low, high and original");
    if (r->factor <= 0 || r->low <= 0 || r->high <= 0 || r->original <= 0) return fail(err, at + "`rot.scaling` must be positive");
    return true;
}

// Sizes and scale of an attention, its window and the first tokens that stay visible behind it.
bool read_windowed(const Json& m, LayerSpec* l, const std::string& at, std::string* err) {
    double scale = 0;
    if (!get_int(m, "heads", &l->heads) || !get_int(m, "kv_heads", &l->kv_heads) || !get_int(m, "dim", &l->dim) || !get_int(m, "vdim", &l->vdim) || !get_num(m, "scale", &scale))
        return fail(err, at + "the mixer needs heads, kv_heads, dim, vdim and scale");
    if (l->heads % l->kv_heads != 0) return fail(err, at + "`kv_heads` does not divide `heads`");
    l->scale = (float)scale;
    l->sink = true;
    const Json* k = m.get("mask");
    if (is_null(k) || !get_int(*k, "size", &l->window)) return fail(err, at + "`mask` needs size");
    if (!get_count(*k, "keep_first", &l->keep_first)) return fail(err, at + "`mask.keep_first` must be a number of tokens");
    return true;
}

// Gebilorn: three kinds of mixers (windowed attention with rotation, windowed attention beside gated linear attention, latent
// attention), mixer and feed-forward in parallel, dense feed-forwards or mixtures with a shared expert, a bigram embedding.
bool read_gebilorn(const Json& j, ModelSpec* s, std::string* err) {
    hm_config& c = s->cfg;
    s->parallel = s->norm_offset = true;
    c.tie_word_embeddings = 1;
    if (!get_int(j, "width", &c.hidden_size) || !get_int(j, "vocab", &c.vocab_size)) return fail(err, "missing `width` or `vocab`");
    const Json *norm = j.get("norm"), *emb = j.get("embedding");
    if (!norm || !get_num(*norm, "eps", &c.rms_norm_eps)) return fail(err, "`norm` needs `eps`");
    double num = 0;
    if (!emb || !get_num(*emb, "scale", &num)) return fail(err, "`embedding` needs `scale`");
    s->embed_scale = (float)num;
    if (const Json* b = emb->get("bigram"); !is_null(b)) {
        double prev = 0, cur = 0;
        int buckets = 0;
        if (!get_int(*b, "buckets", &buckets) || !get_num(*b, "mul_prev", &prev) || !get_num(*b, "mul_cur", &cur) || prev < 0 || cur < 0 || prev > 2147483647.0 || cur > 2147483647.0)
            return fail(err, "`embedding.bigram` needs buckets, mul_prev and mul_cur");
        s->bigram_buckets = buckets;
        s->bigram_prev = (long long)prev;
        s->bigram_cur = (long long)cur;
    }
    const Json* cap = j.get("logit_softcap");
    if (!is_null(cap)) {
        if (!get_num(j, "logit_softcap", &num) || num <= 0) return fail(err, "`logit_softcap` must be positive");
        s->softcap = (float)num;
    }
    const Json* list = j.get("layers");
    if (!list || list->kind != Json::Arr || list->arr.empty()) return fail(err, "missing `layers`");
    for (size_t i = 0; i < list->arr.size(); ++i) {
        const Json& e = list->arr[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        LayerSpec l;
        std::string type, kind;
        const Json *m = e.get("mixer"), *mlp = e.get("mlp");
        if (!get_str(e, "type", &type) || is_null(m)) return fail(err, at + "missing `type` or `mixer`");
        if (type == "attention") {
            l.mixer = MIX_GQA;
            l.qk_norm = QKN_UNIT;
            l.out_gate = GATE_ELEM;
            if (!read_windowed(*m, &l, at, err) || !read_rotation(*m, l.dim, &l.rot, at, err)) return false;
        } else if (type == "parallel") {
            l.mixer = MIX_PARALLEL;
            l.out_gate = GATE_HEAD;
            l.qkv_bias = true;
            const Json *left = m->get("left"), *right = m->get("right");
            double ls = 0, rs = 0, tau = 0;
            if (is_null(left) || is_null(right) || !get_num(*m, "left_scale", &ls) || !get_num(*m, "right_scale", &rs)) return fail(err, at + "the mixer needs left, right, left_scale and right_scale");
            if (!read_windowed(*left, &l, at, err)) return false;
            if (!get_count(*left, "conv", &l.conv)) return fail(err, at + "`left.conv` must be a number of taps");
            if (!get_int(*right, "heads", &l.lin_heads) || !get_int(*right, "dim", &l.lin_dim) || !get_int(*right, "vdim", &l.lin_vdim) || !get_num(*right, "tau", &tau) || tau <= 0)
                return fail(err, at + "`right` needs heads, dim, vdim and tau");
            l.lin_tau = (float)tau;
            l.left_scale = (float)ls;
            l.right_scale = (float)rs;
        } else if (type == "latent_attention") {
            l.mixer = MIX_LATENT;
            if (!get_int(*m, "heads", &l.heads) || !get_int(*m, "dim", &l.dim) || !get_int(*m, "vdim", &l.vdim) || !get_int(*m, "kv_rank", &l.kv_rank) || !get_int(*m, "q_rank", &l.q_rank) ||
                !get_int(*m, "rot_dim", &l.rot_dim) || !get_num(*m, "scale", &num))
                return fail(err, at + "the mixer needs heads, dim, rot_dim, vdim, q_rank, kv_rank and scale");
            l.scale = (float)num;
            if (!read_rotation(*m, l.rot_dim, &l.rot, at, err)) return false;
            if (l.rot.dims != l.rot_dim) return fail(err, at + "`rot.dims` differs from `rot_dim`");
        } else {
            return fail(err, at + "unknown mixer type");
        }
        if (!is_null(mlp)) {
            if (!get_str(*mlp, "kind", &kind)) return fail(err, at + "unknown mlp");
            if (kind == "dense") {
                l.mlp = MLP_GLU;
                l.act = GLU_GELU;
                if (!get_int(*mlp, "ff", &l.ff)) return fail(err, at + "`mlp` needs ff");
            } else if (kind == "moe") {
                const Json *ex = mlp->get("expert"), *r = mlp->get("router"), *sh = mlp->get("shared");
                l.mlp = MLP_MOE;
                l.act = GLU_SILU;
                if (is_null(ex) || !get_int(*ex, "ff", &l.ff)) return fail(err, at + "`mlp.expert` needs ff");
                if (is_null(r) || !get_int(*r, "experts", &l.experts) || !get_int(*r, "top", &l.top) || !get_num(*r, "scale", &num)) return fail(err, at + "`mlp.router` needs experts, top and scale");
                if (l.top > l.experts) return fail(err, at + "`mlp.router.top` is larger than the number of experts");
                l.router_scale = (float)num;
                if (!is_null(sh) && !get_int(*sh, "ff", &l.shared_ff)) return fail(err, at + "`mlp.shared` needs ff");
            } else {
                return fail(err, at + "unknown mlp");
            }
        }
        c.num_attention_heads = std::max(c.num_attention_heads, l.heads);
        c.num_key_value_heads = std::max(c.num_key_value_heads, std::max(l.kv_heads, 1));
        c.head_dim = std::max(c.head_dim, l.dim + l.rot_dim);
        c.intermediate_size = std::max(c.intermediate_size, std::max(l.ff, l.shared_ff));
        s->layers.push_back(l);
    }
    c.num_hidden_layers = (int)s->layers.size();
    c.max_position_embeddings = 1 << 30;  // rotations are computed: the cache is the only limit
    c.intermediate_size = std::max(c.intermediate_size, 1);
    return true;
}

bool read_mask(const Json& m, int* size, const std::string& at, std::string* err) {
    const Json* k = m.get("mask");
    return (!is_null(k) && get_int(*k, "size", size)) || fail(err, at + "`mask` needs size");
}

// Retention: linear attention with a fixed decay per head.
bool read_retention(const Json& m, LayerSpec* l, const std::string& at, std::string* err) {
    l->mixer = MIX_LINEAR;
    l->lin_kind = LIN_RETENTION;
    if (!get_int(m, "heads", &l->lin_heads) || !get_int(m, "dim", &l->lin_dim) || !get_int(m, "vdim", &l->lin_vdim)) return fail(err, at + "the mixer needs heads, dim and vdim");
    l->lin_kv_heads = l->lin_heads;
    const Json* d = m.get("decay");
    if (!d || d->kind != Json::Arr || (int)d->arr.size() != l->lin_heads) return fail(err, at + "`decay` needs a number per head");
    for (const Json& v : d->arr) {
        if (v.kind != Json::Num) return fail(err, at + "`decay` needs a number per head");
        l->lin_decay.push_back((float)v.num);
    }
    return read_rotation(m, l->lin_dim, &l->rot, at, err);
}

// Attention inside chunks whose heads mix their scores, beside the gated delta rule.
bool read_talking_delta(const Json& m, LayerSpec* l, const std::string& at, std::string* err) {
    const Json *left = m.get("left"), *right = m.get("right");
    double scale = 0;
    l->mixer = MIX_PARALLEL;
    l->lin_kind = LIN_DELTA;
    l->tied_values = l->talking = l->sink = true;
    l->out_gate = GATE_ELEM;
    if (is_null(left) || is_null(right)) return fail(err, at + "the mixer needs left and right");
    if (!get_int(*left, "heads", &l->heads) || !get_int(*left, "kv_heads", &l->kv_heads) || !get_int(*left, "dim", &l->dim) || !get_int(*left, "vdim", &l->vdim) || !get_num(*left, "scale", &scale))
        return fail(err, at + "`left` needs heads, kv_heads, dim, vdim and scale");
    if (l->heads % l->kv_heads != 0) return fail(err, at + "`left.kv_heads` does not divide `left.heads`");
    if (l->vdim != l->dim) return fail(err, at + "`left.vdim` differs from `left.dim`: the values are the keys");
    l->scale = (float)scale;
    if (!get_int(*left, "conv", &l->conv)) return fail(err, at + "`left.conv` must be a number of taps");
    if (!read_mask(*left, &l->chunk, at, err) || !read_rotation(*left, l->dim, &l->rot, at, err)) return false;
    if (!get_int(*right, "heads", &l->lin_heads) || !get_int(*right, "kv_heads", &l->lin_kv_heads) || !get_int(*right, "dim", &l->lin_dim) || !get_int(*right, "vdim", &l->lin_vdim))
        return fail(err, at + "`right` needs heads, kv_heads, dim and vdim");
    if (l->lin_heads % l->lin_kv_heads != 0) return fail(err, at + "`right.kv_heads` does not divide `right.heads`");
    return get_int(*right, "conv", &l->lin_conv) || fail(err, at + "`right.conv` must be a number of taps");
}

// Latent attention with a rotated part inside a window; a layer may read the latents of an earlier one.
bool read_windowed_latent(const Json& m, const ModelSpec& s, LayerSpec* l, const std::string& at, std::string* err) {
    double scale = 0;
    l->mixer = MIX_LATENT;
    l->out_gate = GATE_HEAD;
    if (!get_int(m, "heads", &l->heads) || !get_int(m, "dim", &l->dim) || !get_int(m, "vdim", &l->vdim) || !get_int(m, "kv_rank", &l->kv_rank) || !get_int(m, "rot_dim", &l->rot_dim) || !get_num(m, "scale", &scale))
        return fail(err, at + "the mixer needs heads, dim, rot_dim, vdim, kv_rank and scale");
    l->scale = (float)scale;
    if (!read_mask(m, &l->window, at, err) || !read_rotation(m, l->rot_dim, &l->rot, at, err)) return false;
    if (l->rot.dims != l->rot_dim) return fail(err, at + "`rot.dims` differs from `rot_dim`");
    const Json* from = m.get("kv_from");
    if (is_null(from)) return true;
    if (from->kind != Json::Num || from->num < 0 || from->num != std::floor(from->num) || from->num >= (double)s.layers.size()) return fail(err, at + "`kv_from` must name an earlier layer");
    l->kv_from = (int)from->num;
    const LayerSpec& o = s.layers[l->kv_from];
    if (o.mixer != MIX_LATENT || o.kv_from >= 0) return fail(err, at + "`kv_from` names a layer without latents of its own");
    if (o.kv_rank != l->kv_rank || o.rot_dim != l->rot_dim) return fail(err, at + "`kv_from` names a layer of another kv_rank or rot_dim");
    return true;
}

// Pulenex: layer norms in front of and behind every sublayer; retention, chunked attention with talking heads beside the gated delta
// rule, windowed latent attention; clamped gated feed-forwards with biases (or none).
bool read_pulenex(const Json& j, ModelSpec* s, std::string* err) {
    hm_config& c = s->cfg;
    s->sandwich = true;
    double num = 0;
    if (!get_int(j, "width", &c.hidden_size) || !get_int(j, "vocab", &c.vocab_size)) return fail(err, "missing `width` or `vocab`");
    const Json *norm = j.get("norm"), *list = j.get("layers");
    if (!norm || !get_num(*norm, "eps", &c.rms_norm_eps)) return fail(err, "`norm` needs `eps`");
    if (!get_num(j, "logit_scale", &num)) return fail(err, "missing `logit_scale`");
    s->logit_scale = (float)num;
    if (!list || list->kind != Json::Arr || list->arr.empty()) return fail(err, "missing `layers`");
    for (size_t i = 0; i < list->arr.size(); ++i) {
        const Json& e = list->arr[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        LayerSpec l;
        std::string type, kind;
        const Json *m = e.get("mixer"), *mlp = e.get("mlp");
        if (!get_str(e, "type", &type) || is_null(m)) return fail(err, at + "missing `type` or `mixer`");
        if (type == "retention") {
            if (!read_retention(*m, &l, at, err)) return false;
        } else if (type == "parallel") {
            if (!read_talking_delta(*m, &l, at, err)) return false;
        } else if (type == "latent_attention") {
            if (!read_windowed_latent(*m, *s, &l, at, err)) return false;
        } else {
            return fail(err, at + "unknown mixer type");
        }
        if (!is_null(mlp)) {
            if (!get_str(*mlp, "kind", &kind) || kind != "dense") return fail(err, at + "unknown mlp");
            l.mlp = MLP_GLU;
            l.act = GLU_CLAMPED;
            l.mlp_bias = true;
            if (!get_int(*mlp, "ff", &l.ff) || !get_num(*mlp, "limit", &num)) return fail(err, at + "`mlp` needs ff and limit");
            l.limit = (float)num;
        }
        c.num_attention_heads = std::max(c.num_attention_heads, std::max(l.heads, l.lin_heads));
        c.num_key_value_heads = std::max(c.num_key_value_heads, std::max(l.kv_heads, 1));
        c.head_dim = std::max(c.head_dim, std::max(l.dim + l.rot_dim, l.lin_dim));
        c.intermediate_size = std::max(c.intermediate_size, l.ff);
        s->layers.push_back(l);
    }
    c.num_hidden_layers = (int)s->layers.size();
    c.max_position_embeddings = 1 << 30;  // rotations are computed: the cache is the only limit
    c.intermediate_size = std::max(c.intermediate_size, 1);
    return true;
}

struct Design {
    const char* name;
    bool (*read)(const Json&, ModelSpec*, std::string*);
};
const Design kDesigns[] = {{"Tunitar", read_tunitar}, {"Dipisun", read_dipisun}, {"Gebilorn", read_gebilorn}, {"Pulenex", read_pulenex}};

}  // namespace

std::vector<double> rotation_turns(const RotSpec& r) {
    const double full = 6.283185307179586;
    std::vector<double> t(r.dims / 2);
    for (size_t i = 0; i < t.size(); ++i) {
        const double f = std::pow(r.base, -2.0 * (double)i / r.dims), wave = full / f;
        double turned = f;
        if (r.scaled && wave > r.original / r.low) {
            turned = f / r.factor;
        } else if (r.scaled && wave >= r.original / r.high) {
            const double s = (r.original / wave - r.low) / (r.high - r.low);
            turned = (1.0 - s) * f / r.factor + s * f;
        }
        t[i] = turned / full;
    }
    return t;
}

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

namespace {
std::string parallel_layer_json(const LayerSpec& l) {
    std::string o;
    char t[768];
    auto rot = [&]() {
        std::snprintf(t, sizeof(t), ",\"rot\":{\"dims\":%d,\"base\":%.9g", l.rot.dims, l.rot.base);
        o += t;
        if (l.rot.scaled) {
            std::snprintf(t, sizeof(t), ",\"factor\":%.9g,\"low\":%.9g,\"high\":%.9g,\"original\":%.9g", l.rot.factor, l.rot.low, l.rot.high, l.rot.original);
            o += t;
        }
        o += "}";
    };
    if (l.mixer == MIX_LATENT) {
        std::snprintf(t, sizeof(t), "{\"type\":\"latent_attention\",\"heads\":%d,\"dim\":%d,\"rot_dim\":%d,\"vdim\":%d,\"q_rank\":%d,\"kv_rank\":%d,\"scale\":%.9g", l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.scale);
        o += t;
        rot();
    } else {
        std::snprintf(t, sizeof(t), "{\"type\":\"%s\",\"heads\":%d,\"kv_heads\":%d,\"dim\":%d,\"vdim\":%d,\"scale\":%.9g,\"window\":%d,\"keep_first\":%d,\"conv\":%d", l.mixer == MIX_GQA ? "windowed_attention" : "parallel", l.heads, l.kv_heads,
                      l.dim, l.vdim, l.scale, l.window, l.keep_first, l.conv);
        o += t;
        if (l.rot.dims) rot();
        if (l.mixer == MIX_PARALLEL) {
            std::snprintf(t, sizeof(t), ",\"linear\":{\"heads\":%d,\"dim\":%d,\"vdim\":%d,\"tau\":%.9g},\"left_scale\":%.9g,\"right_scale\":%.9g", l.lin_heads, l.lin_dim, l.lin_vdim, l.lin_tau, l.left_scale, l.right_scale);
            o += t;
        }
    }
    std::snprintf(t, sizeof(t), ",\"ff\":%d,\"experts\":%d,\"top\":%d,\"router_scale\":%.9g,\"shared_ff\":%d}", l.ff, l.experts, l.top, l.router_scale, l.shared_ff);
    return o + t;
}
std::string sandwich_layer_json(const LayerSpec& l) {
    char t[768];
    std::string o = "{\"type\":\"";
    auto put = [&](const char* f, auto... v) {
        std::snprintf(t, sizeof(t), f, v...);
        o += t;
    };
    auto rot = [&]() { put(",\"rot\":{\"dims\":%d,\"base\":%.9g}", l.rot.dims, l.rot.base); };
    if (l.mixer == MIX_LINEAR) {
        put("retention\",\"heads\":%d,\"dim\":%d,\"vdim\":%d", l.lin_heads, l.lin_dim, l.lin_vdim);
        o += ",\"decay\":[";
        for (size_t i = 0; i < l.lin_decay.size(); ++i) put(i ? ",%.9g" : "%.9g", l.lin_decay[i]);
        o += "]";
    } else if (l.mixer == MIX_LATENT) {
        put("latent_attention\",\"heads\":%d,\"dim\":%d,\"rot_dim\":%d,\"vdim\":%d,\"kv_rank\":%d,\"scale\":%.9g,\"window\":%d,\"kv_from\":%s", l.heads, l.dim, l.rot_dim, l.vdim, l.kv_rank, l.scale, l.window,
            l.kv_from < 0 ? "null" : std::to_string(l.kv_from).c_str());
    } else {
        put("parallel\",\"heads\":%d,\"kv_heads\":%d,\"dim\":%d,\"vdim\":%d,\"scale\":%.9g,\"chunk\":%d,\"conv\":%d", l.heads, l.kv_heads, l.dim, l.vdim, l.scale, l.chunk, l.conv);
        put(",\"linear\":{\"heads\":%d,\"kv_heads\":%d,\"dim\":%d,\"vdim\":%d,\"conv\":%d}", l.lin_heads, l.lin_kv_heads, l.lin_dim, l.lin_vdim, l.lin_conv);
    }
    rot();
    put(",\"ff\":%d,\"limit\":%.9g}", l.ff, l.limit);
    return o;
}
}  // namespace

std::string layers_json(const ModelSpec& spec) {
    std::string o = "[";
    for (size_t i = 0; i < spec.layers.size(); ++i) {
        const LayerSpec& l = spec.layers[i];
        char t[768];
        if (i) o += ",";
        if (spec.parallel || spec.sandwich) {
            o += spec.parallel ? parallel_layer_json(l) : sandwich_layer_json(l);
            continue;
        }
        if (l.mixer == MIX_LATENT) {
            std::snprintf(t, sizeof(t), "{\"type\":\"latent_attention\",\"heads\":%d,\"dim\":%d,\"vdim\":%d,\"kv_rank\":%d,\"kv_from\":%s,\"scale\":%.9g,\"ff\":%d}", l.heads, l.dim, l.vdim, l.kv_rank,
                          l.kv_from < 0 ? "null" : std::to_string(l.kv_from).c_str(), l.scale, l.ff);
            o += t;
            continue;
        }
        std::snprintf(t, sizeof(t), "{\"type\":\"grouped_attention\",\"heads\":%d,\"kv_heads\":%d,\"dim\":%d,\"vdim\":%d,\"scale\":%.9g,\"qk_norm\":\"%s\",\"temp_coef\":%.9g,\"temp_every\":%d,\"bias_reach\":%.9g,\"v_first\":%s", l.heads,
                      l.kv_heads, l.dim, l.vdim, l.scale, l.qk_norm == QKN_ALL ? "all" : l.qk_norm == QKN_HEAD ? "head" : "none", l.temp_coef, l.temp_every, l.bias_reach, l.v_first < 0 ? "null" : std::to_string(l.v_first).c_str());
        o += t;
        std::snprintf(t, sizeof(t), ",\"ff\":%d,\"experts\":%d,\"identity\":%d,\"top\":%d,\"limit\":%.9g}", l.ff, l.experts, l.identity, l.top, l.limit);
        o += t;
    }
    return o + "]";
}

}  // namespace hm
