// Engine parts for listed designs whose sublayers stand between two layer norms: weights, scratch, and the launches of one layer.
// Beside engine_listed.cu, engine_gqa.cu and engine_parallel.cu, whose attention kernels and pieces they use.
//
// A layer is, per pass,
//   in     [everything that the mixer reads off its normed input]; queries and keys that need no convolution leave rotated
//   side   convolutions, rotations, page slots; latents; rows for the recurrence                                  (side.cu)
//   recur  linear attention                                                                                      (recur.cu)
//   attn   softmax attention with its output gate
//   out    output projection (two of them side by side in parallel mixers)
//   norm   residual += norm(result), and the norm that the next projection reads                                 (sandwich.cu)
//   gate and up, down, norm
// Layers of linear attention alone have neither side nor attn; latent attention has key up and value up around attn.
#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <cstring>

#include "engine_parallel.h"
#include "engine_util.h"
#include "gemm_tc.h"
#include "recur.h"
#include "sandwich.h"

namespace hm {

namespace {
// Retention: columns from one head's queries (or keys) to the next; rotated pairs lie side by side in front, zeros fill up.
int lin_stride(const LayerSpec& s) { return gla_pad(s.lin_dim); }
int round64(int n) { return (n + 63) / 64 * 64; }
int glu_blocks(int ff) { return (ff + 63) / 64; }

// Rows of a pass that are prepared for a recurrence, in floats.
struct PreparedRows {
    size_t q, k, v, alpha, gate, total;
};
PreparedRows prepared_rows(const LayerSpec& s) {
    PreparedRows r{};
    if (s.lin_kind != LIN_DELTA || !s.linear()) return r;
    auto take = [&](size_t n) {
        const size_t first = r.total;
        r.total += TC_ROWS * n;
        return first;
    };
    r.q = take((size_t)s.lin_kv_heads * s.lin_dim);
    r.k = take((size_t)s.lin_kv_heads * s.lin_dim);
    r.v = take((size_t)s.lin_heads * s.lin_vdim);
    r.alpha = take((size_t)s.lin_heads * s.lin_dim);
    r.gate = take((size_t)s.lin_heads * s.lin_vdim);
    return r;
}
}  // namespace

ParallelColumns sandwich_columns(const LayerSpec& s) {
    ParallelColumns c;
    int at = 0;
    auto take = [&](int n) {
        const int first = at;
        at += (n + 7) / 8 * 8;
        return first;
    };
    if (s.mixer == MIX_LINEAR) {
        c.lq = take(2 * s.lin_heads * lin_stride(s));
        c.lk = c.lq + s.lin_heads * lin_stride(s);
        c.lv = take(s.lin_heads * s.lin_vdim);
        c.lg = take(s.lin_heads * s.lin_vdim);
        c.k_out = round64(s.lin_heads * s.lin_vdim);
    } else if (s.mixer == MIX_LATENT) {
        c.q = take(s.heads * s.q_stride());
        if (s.kv_from < 0) c.dkv = take(s.latent_rank());
        c.gates = s.heads;
        c.gate = take(c.gates);
        c.k_out = round64(s.heads * s.vdim);
    } else {
        c.q = take((s.heads + s.kv_heads) * s.dim);
        c.k = c.q + s.heads * s.dim;
        c.gates = s.heads * s.vdim;
        c.gate = take(c.gates);
        c.lq = take(s.lin_channels());
        c.lk = c.lq + s.lin_kv_heads * s.lin_dim;
        c.lv = c.lk + s.lin_kv_heads * s.lin_dim;
        c.lb = take(s.lin_heads);
        c.la = take(s.decay_rank);
        c.lgl = take(s.gate_rank);
        c.k_out = std::max(round64(s.heads * s.vdim), round64(s.lin_heads * s.lin_vdim));  // of either of the two output projections
    }
    c.ff = s.ff;
    c.n = c.ld = at;
    return c;
}

// ---- weights -------------------------------------------------------------------------------------

// Group `g` of a grouped projection whose groups come as tensors of their own, with at most K inputs.
int Engine::load_group(LinearW& L, int groups, int g, int K, int k_part, int group_n, int dtype, const void* host, size_t nbytes) {
    if (dtype != HM_BF16) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
    if (nbytes != (size_t)group_n * k_part * 2) return fail(HM_ERR_INVALID, "tensor byte size does not match its shape");
    L.K = K;
    L.groups = groups;
    L.group_n = group_n;
    L.group_slabs = (group_n + SLAB - 1) / SLAB;
    L.N = groups * group_n;
    L.kind = HM_BF16;
    cfg_.weight_dtype = HM_BF16;
    auto room = [&](uint16_t** p, size_t bytes) -> cudaError_t {
        if (*p) return cudaSuccess;
        const cudaError_t e = cudaMalloc(p, bytes);
        return e == cudaSuccess ? cudaMemsetAsync(*p, 0, bytes, stream_) : e;
    };
    void* tmp = nullptr;
    const int rc = stage(host, nbytes, &tmp);
    if (rc) return rc;
    const uint16_t* src = static_cast<const uint16_t*>(tmp);
    const int n_off = g * L.group_slabs * SLAB;
    cudaError_t ce = room(&L.slabs, (size_t)L.columns() * K * 2);
    if (ce == cudaSuccess) ce = launch_pack_slabs_from_nk(src, group_n, k_part, L.slabs, n_off, -1, stream_, K, 0);
    if (use_tc_) {
        if (ce == cudaSuccess) ce = room(&L.tc, tc_packed_elems(K, L.columns()) * 2);
        if (ce == cudaSuccess) ce = launch_pack_tc(src, group_n, k_part, false, L.tc, n_off, -1, stream_, K, 0);
    }
    if (ce == cudaSuccess) ce = cudaStreamSynchronize(stream_);
    cudaFree(tmp);
    if (ce != cudaSuccess) return cuda_fail(ce, "load_group");
    L.loaded_parts++;
    return HM_OK;
}

int Engine::load_sandwich_tensor(int layer, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    LayerW& w = layers_[layer];
    LayerSpec& s = spec_.layers[layer];
    size_t n = 1;
    for (int i = 0; i < ndim; ++i) n *= (size_t)shape[i];
    auto bad_shape = [&]() { return fail(HM_ERR_INVALID, "unexpected shape for tensor " + name); };
    auto is2 = [&](int64_t a, int64_t b) { return ndim == 2 && shape[0] == a && shape[1] == b; };
    auto unknown = [&]() { return fail(HM_ERR_INVALID, "unknown tensor name: " + name); };
    if (std::find(w.seen.begin(), w.seen.end(), rest) != w.seen.end()) return fail(HM_ERR_STATE, "tensor loaded twice: " + name);
    if (s.lin_kind == LIN_DELTA && (s.decay_rank == 0 || s.gate_rank == 0)) {
        if (ndim == 2) note_shape(name, {shape[0], shape[1]});
        if (s.decay_rank == 0 || s.gate_rank == 0) {  // the sizes of two latents are only in their tensors' shapes: wait for both
            const uint8_t* bytes = static_cast<const uint8_t*>(host);
            w.pending.push_back({name, rest, dtype, {shape, shape + ndim}, {bytes, bytes + nbytes}});
            return HM_OK;
        }
        const std::vector<LayerW::Pending> kept = std::move(w.pending);
        w.pending.clear();
        for (const LayerW::Pending& p : kept)
            if (const int rc = load_sandwich_tensor(layer, p.name, p.rest, p.dtype, p.shape.data(), (int)p.shape.size(), p.data.data(), p.data.size())) return rc;
        if (std::find(w.seen.begin(), w.seen.end(), rest) != w.seen.end()) return fail(HM_ERR_STATE, "tensor loaded twice: " + name);
    }
    const ParallelColumns c = sandwich_columns(s);
    auto bf16 = [&]() { return dtype == HM_BF16 && nbytes == n * 2; };
    const uint16_t* bits = static_cast<const uint16_t*>(host);
    auto in = [&](int off, int part) { return is2(part, H_) ? load_linear(w.in, H_, c.n, off, part, -1, dtype, host, nbytes) : bad_shape(); };
    auto vec = [&](float** dst, size_t len) { return ndim != 1 || n != len ? bad_shape() : load_vec_f32(dst, len, 0, dtype, host, n, nbytes); };
    auto conv = [&](float** dst, size_t total, size_t first, int channels, int taps) { return is2(channels, taps) ? load_vec_f32(dst, total * taps, first * taps, dtype, host, n, nbytes) : bad_shape(); };
    auto to_f32 = [&](size_t i) {
        if (dtype == HM_F32) return static_cast<const float*>(host)[i];
        const uint32_t u = (uint32_t)bits[i] << 16;
        float f;
        std::memcpy(&f, &u, 4);
        return f;
    };
    auto floats = [&](std::vector<float>* v) {
        if ((dtype != HM_BF16 && dtype != HM_F32) || nbytes != n * (dtype == HM_BF16 ? 2 : 4)) return fail(HM_ERR_UNSUPPORTED, name + " must be stored as bf16 or f32");
        v->resize(n);
        for (size_t i = 0; i < n; ++i) (*v)[i] = to_f32(i);
        return (int)HM_OK;
    };
    // [columns, rank] -> [rank][columns]
    auto factor = [&](float** dst, int cols, int rank) {
        if (!is2(cols, rank)) return bad_shape();
        std::vector<float> v, t(n);
        if (const int rc = floats(&v)) return rc;
        for (int i = 0; i < cols; ++i)
            for (int r = 0; r < rank; ++r) t[(size_t)r * cols + i] = v[(size_t)i * rank + r];
        return upload(dst, t);
    };
    // rows of every head to other places: row e of a head of `per` to place(e) of `stride`
    auto placed = [&](int heads, int per, int stride, int off, auto place) {
        if (!is2((int64_t)heads * per, H_)) return bad_shape();
        if (!bf16()) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
        std::vector<uint16_t> m((size_t)heads * stride * H_, 0);
        for (int h = 0; h < heads; ++h)
            for (int e = 0; e < per; ++e) std::memcpy(&m[((size_t)h * stride + place(e)) * H_], bits + ((size_t)h * per + e) * H_, (size_t)H_ * 2);
        return load_linear(w.in, H_, c.n, off, heads * stride, -1, dtype, m.data(), m.size() * 2);
    };
    const int vals = s.heads * s.vdim, lin_vals = s.lin_heads * s.lin_vdim, lin_k = s.lin_heads * s.lin_dim;
    auto retention = [&](const std::string& t) -> int {
        // halves that turn together become neighbours, for queries and keys alike
        const int half = s.rot.dims / 2;
        auto place = [&](int e) { return e < half ? 2 * e : e < 2 * half ? 2 * (e - half) + 1 : e; };
        if (t == "q") return placed(s.lin_heads, s.lin_dim, lin_stride(s), c.lq, place);
        if (t == "k") return placed(s.lin_heads, s.lin_dim, lin_stride(s), c.lk, place);
        if (t == "v") return in(c.lv, lin_vals);
        if (t == "g") return in(c.lg, lin_vals);
        if (t == "o") return is2(H_, lin_vals) ? load_inputs(w.o, c.k_out, 0, lin_vals, H_, dtype, host, nbytes) : bad_shape();
        return unknown();
    };
    auto latent = [&](const std::string& t) -> int {
        const int R = s.latent_rank(), qs = s.q_stride();
        if (t == "q") return placed(s.heads, s.dim + s.rot_dim, qs, c.q, [&](int e) { return e < s.dim ? s.rot_dim + e : e - s.dim; });  // rotated elements first
        if (t == "dkv" && s.kv_from < 0) return in(c.dkv, R);
        if (t == "dkv.norm" && s.kv_from < 0) return vec(&w.latent_norm, s.kv_rank);
        if (t == "g") return in(c.gate, s.heads);
        if (t == "uk") return load_key_up(w, s, name, dtype, shape, ndim, host, nbytes);
        if (t == "uv") return load_value_up(w, s, name, dtype, shape, ndim, host, nbytes);
        if (t == "o") return is2(H_, vals) ? load_inputs(w.o, c.k_out, 0, vals, H_, dtype, host, nbytes) : bad_shape();
        return unknown();
    };
    auto left = [&](const std::string& t) -> int {
        const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim;
        if (t == "q") return in(c.q, nq);
        if (t == "k") return in(c.k, nk);
        if (t == "q.conv" && s.conv > 0) return conv(&w.conv_w, nq + nk, 0, nq, s.conv);
        if (t == "k.conv" && s.conv > 0) return conv(&w.conv_w, nq + nk, nq, nk, s.conv);
        if (t == "talk") return is2(s.heads, s.heads) ? load_vec_f32(&w.talk, n, 0, dtype, host, n, nbytes) : bad_shape();
        if (t == "temp") return vec(&w.temp, s.heads);
        if (t == "sink") return vec(&w.sink, s.heads);
        if (t == "g") return in(c.gate, vals);
        if (t == "o") return is2(H_, vals) ? load_group(w.o, 2, 0, c.k_out, vals, H_, dtype, host, nbytes) : bad_shape();
        if (t == "out") return vec(&w.left_out, H_);
        return unknown();
    };
    auto right = [&](const std::string& t) -> int {
        const int nk = s.lin_kv_heads * s.lin_dim, ch = s.lin_channels();
        if (t == "q") return in(c.lq, nk);
        if (t == "k") return in(c.lk, nk);
        if (t == "v") return in(c.lv, lin_vals);
        if (t == "q.conv" && s.lin_conv > 0) return conv(&w.lin_conv_w, ch, 0, nk, s.lin_conv);
        if (t == "k.conv" && s.lin_conv > 0) return conv(&w.lin_conv_w, ch, nk, nk, s.lin_conv);
        if (t == "v.conv" && s.lin_conv > 0) return conv(&w.lin_conv_w, ch, 2 * nk, lin_vals, s.lin_conv);
        if (t == "b") return in(c.lb, s.lin_heads);
        if (t == "a1") return in(c.la, s.decay_rank);
        if (t == "g1") return in(c.lgl, s.gate_rank);
        if (t == "a2") return factor(&w.lin_up, lin_k, s.decay_rank);
        if (t == "g2") return factor(&w.lin_up_g, lin_vals, s.gate_rank);
        if (t == "dt_bias") return vec(&w.lin_bias, lin_k);
        if (t == "norm") return vec(&w.lin_norm, s.lin_vdim);
        if (t == "o") return is2(H_, lin_vals) ? load_group(w.o, 2, 1, c.k_out, lin_vals, H_, dtype, host, nbytes) : bad_shape();
        if (t == "out") return vec(&w.right_out, H_);
        if (t != "A_log") return unknown();
        if (ndim != 1 || n != (size_t)s.lin_heads) return bad_shape();
        std::vector<float> v;
        if (const int rc = floats(&v)) return rc;
        for (float& x : v) x = (float)-std::exp((double)x);
        return upload(&w.lin_rate, v);
    };
    auto feed_forward = [&](const std::string& t) -> int {
        if (s.mlp != MLP_GLU) return unknown();
        const int blocks = glu_blocks(s.ff);
        for (int part = 0; part < 2; ++part) {
            const std::string p = part ? "up" : "gate";
            if (t == p) return is2(s.ff, H_) ? load_linear(w.gu, H_, blocks * SLAB, 0, s.ff, part, dtype, host, nbytes) : bad_shape();
            if (t != p + ".b") continue;
            if (ndim != 1 || n != (size_t)s.ff) return bad_shape();
            std::vector<float> v;
            if (const int rc = floats(&v)) return rc;
            w.gu_bias_host.resize((size_t)blocks * SLAB, 0.f);
            for (int i = 0; i < s.ff; ++i) w.gu_bias_host[(size_t)(i / 64) * SLAB + part * 64 + i % 64] = v[i];
            return HM_OK;
        }
        if (t == "down") return is2(H_, s.ff) ? load_linear(w.down, s.ff, H_, 0, H_, -1, dtype, host, nbytes) : bad_shape();
        if (t == "down.b") return vec(&w.down_bias, H_);
        return unknown();
    };
    int rc;
    if (rest == "norm1b") rc = vec(&w.norm1b, H_);
    else if (rest == "norm2" && s.mlp != MLP_NONE) rc = vec(&w.post_ln, H_);
    else if (rest == "norm2b" && s.mlp != MLP_NONE) rc = vec(&w.norm2b, H_);
    else if (rest.compare(0, 4, "mlp.") == 0) rc = feed_forward(rest.substr(4));
    else if (s.mixer == MIX_PARALLEL && rest.compare(0, 9, "mix.left.") == 0) rc = left(rest.substr(9));
    else if (s.mixer == MIX_PARALLEL && rest.compare(0, 10, "mix.right.") == 0) rc = right(rest.substr(10));
    else if (s.mixer == MIX_LINEAR && rest.compare(0, 4, "mix.") == 0) rc = retention(rest.substr(4));
    else if (s.mixer == MIX_LATENT && rest.compare(0, 4, "mix.") == 0) rc = latent(rest.substr(4));
    else rc = unknown();
    if (rc == HM_OK) w.seen.push_back(rest);
    return rc;
}

int Engine::finalize_sandwich() {
    for (int l = 0; l < L_; ++l) {
        LayerW& w = layers_[l];
        const LayerSpec& s = spec_.layers[l];
        std::vector<std::string> need = {"norm1b"};
        auto all = [&](const std::string& p, std::initializer_list<const char*> names) {
            for (const char* t : names) need.push_back(p + t);
        };
        if (s.mixer == MIX_LINEAR) all("mix.", {"q", "k", "v", "g", "o"});
        if (s.mixer == MIX_LATENT) {
            all("mix.", {"q", "uk", "uv", "g", "o"});
            if (s.kv_from < 0) all("mix.", {"dkv", "dkv.norm"});
        }
        if (s.mixer == MIX_PARALLEL) {
            all("mix.left.", {"q", "k", "talk", "temp", "sink", "g", "o", "out"});
            if (s.conv > 0) all("mix.left.", {"q.conv", "k.conv"});
            all("mix.right.", {"q", "k", "v", "b", "A_log", "norm", "a1", "a2", "dt_bias", "g1", "g2", "o", "out"});
            if (s.lin_conv > 0) all("mix.right.", {"q.conv", "k.conv", "v.conv"});
        }
        if (s.mlp == MLP_GLU) all("", {"norm2", "norm2b", "mlp.gate", "mlp.gate.b", "mlp.up", "mlp.up.b", "mlp.down", "mlp.down.b"});
        const std::string at = "missing weight in layer " + std::to_string(l) + ": ";
        if (!w.in_ln) return fail(HM_ERR_STATE, at + "norm1");
        for (const std::string& t : need)
            if (std::find(w.seen.begin(), w.seen.end(), t) == w.seen.end()) return fail(HM_ERR_STATE, at + t);
        if (!w.gu_bias_host.empty()) {
            const int rc = upload(&w.gu_bias, w.gu_bias_host);
            if (rc) return rc;
        }
        if (s.lin_kind == LIN_RETENTION) {
            const int rc = upload(&w.lin_decay, s.lin_decay);
            if (rc) return rc;
        }
        if (s.rot.dims) {
            const std::vector<double> t = rotation_turns(s.rot);
            HM_CUDA(cudaMalloc(&w.turns, t.size() * 8));
            HM_CUDA(cudaMemcpy(w.turns, t.data(), t.size() * 8, cudaMemcpyHostToDevice));
        }
    }
    // logits are linear in the final norm's weight
    std::vector<float> f(H_);
    HM_CUDA(cudaMemcpy(f.data(), final_norm_, H_ * 4, cudaMemcpyDeviceToHost));
    for (float& x : f) x *= spec_.logit_scale;
    HM_CUDA(cudaMemcpy(final_norm_, f.data(), H_ * 4, cudaMemcpyHostToDevice));
    return HM_OK;
}

// ---- scratch ---------------------------------------------------------------------------------------

int Engine::alloc_sandwich_scratch() {
    if (!spec_.sandwich) return HM_OK;
    size_t prep = 1;
    int k_out = 1;
    cat_ld_ = 1;
    for (const LayerSpec& s : spec_.layers) {
        prep = std::max(prep, prepared_rows(s).total);
        const int k = sandwich_columns(s).k_out;
        k_out = std::max(k_out, k * (s.mixer == MIX_PARALLEL ? 2 : 1));
    }
    auto get = [&](auto** p, size_t count) -> cudaError_t {
        const cudaError_t e = cudaMalloc((void**)p, count * sizeof(**p));
        return e == cudaSuccess ? cudaMemset(*p, 0, count * sizeof(**p)) : e;
    };
    cat_ld_ = k_out;
    HM_CUDA(get(&normed_, (size_t)TC_ROWS * H_));
    HM_CUDA(get(&cat_, (size_t)TC_ROWS * k_out));
    HM_CUDA(get(&sub_, (size_t)TC_ROWS * 2 * H_));
    HM_CUDA(get(&lin_rows_, prep));
    if (use_tc_) HM_CUDA(get(&xpack_cat_, tc_xpack_bytes(TC_ROWS, k_out)));
    return HM_OK;
}

// ---- one layer ---------------------------------------------------------------------------------------

// residual += norm(what the sublayer left in sub_) unless post_w is null, and the residual's norm for the projection behind
int Engine::enqueue_sandwich(int M, bool tall, const LayerW* joined, const float* post_w, const float* next_w, int* launches) {
    if (only_class_ >= 0 && only_class_ != PC_NORM) return HM_OK;
    SandwichArgs a{};
    a.x = h_;
    a.y = post_w ? sub_ : nullptr;
    a.ldy = H_;
    if (joined) {
        a.ldy = 2 * H_;
        a.left_w = joined->left_out;
        a.right_w = joined->right_out;
    }
    a.w = post_w;
    a.next_w = next_w;
    a.eps = (float)cfg_.rms_norm_eps;
    a.M = M;
    a.W = H_;
    a.normed = normed_;
    if (tall) {
        a.xp = xpack_;
        a.xp_mpad = tc_mpad(M);
    }
    const cudaError_t ce = launch_sandwich(a, stream_, pdl_);
    if (ce != cudaSuccess) return cuda_fail(ce, "norm launch");
    ++*launches;
    return HM_OK;
}

SideArgs Engine::sandwich_side_args(int l, int M, const int32_t* row_pos, const int32_t* row_seq) const {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    const ParallelColumns c = sandwich_columns(s);
    SideArgs a{};
    a.M = M;
    a.ld = c.ld;
    a.xp_mpad = tc_mpad(M);
    a.eps = (float)cfg_.rms_norm_eps;
    a.row_pos = row_pos;
    a.row_seq = row_seq;
    if (s.mixer == MIX_LATENT) {
        a.has_latent = 1;
        a.latent.pool = latent_pool(l);
        a.latent.c = mix_raw_ + c.dkv;
        a.latent.w = w.latent_norm;
        a.latent.rot_pairs = s.rot_dim / 2;
        a.latent.turns = w.turns;
        a.latent.neighbours = 1;
        return a;
    }
    int longest = 1;
    const GqaRuns runs = pass_runs(M, &longest);
    const PreparedRows r = prepared_rows(s);
    GqaPostArgs p{};
    p.ld = c.ld;
    p.M = M;
    p.row_pos = row_pos;
    p.row_seq = row_seq;
    p.runs = runs;
    p.conv_stride = state_floats_;
    a.has_post = a.has_post2 = a.has_low = 1;
    a.post = a.post2 = p;
    GqaPostArgs& t = a.post;
    t.pool = gqa_pool(l);
    t.raw = mix_raw_ + c.q;
    t.heads = s.heads;
    t.q_scale = (float)(s.scale * 1.4426950408889634);
    t.head_scale = w.temp;
    t.q_out = q_;
    t.taps = s.conv;
    t.conv_w = w.conv_w;
    t.conv_state = state_ ? state_ + w.conv_at : nullptr;
    t.rot_dims = s.rot.dims;
    t.rot_neighbours = 1;
    t.turns = w.turns;
    t.tied_values = 1;
    GqaPostArgs& d = a.post2;
    d.pool.kv_heads = s.lin_kv_heads;
    d.pool.dim = s.lin_dim;
    d.pool.vdim = s.lin_vdim;
    d.raw = mix_raw_ + c.lq;
    d.heads = s.lin_kv_heads;
    d.v_heads = s.lin_heads;
    d.qk_norm = QKN_SUM;
    d.eps = 1e-6f;
    d.q_scale = 1.0f / std::sqrt((float)s.lin_dim);
    d.q_out = lin_rows_ + r.q;
    d.k_out = lin_rows_ + r.k;
    d.v_out = lin_rows_ + r.v;
    d.taps = s.lin_conv;
    d.conv_w = w.lin_conv_w;
    d.conv_state = state_ ? state_ + w.lin_conv_at : nullptr;
    d.conv_silu = 1;
    LowRankSide& f = a.low;
    f.a = mix_raw_ + c.la;
    f.g = mix_raw_ + c.lgl;
    f.rank_a = s.decay_rank;
    f.rank_g = s.gate_rank;
    f.up_a = w.lin_up;
    f.bias = w.lin_bias;
    f.neg_rate = w.lin_rate;
    f.up_g = w.lin_up_g;
    f.heads = s.lin_heads;
    f.dim = s.lin_dim;
    f.vdim = s.lin_vdim;
    f.alpha = lin_rows_ + r.alpha;
    f.gate = lin_rows_ + r.gate;
    return a;
}

RecurArgs Engine::recur_args(int l, int M, bool tall, const int32_t* row_pos, const int32_t* row_seq) const {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    const ParallelColumns c = sandwich_columns(s);
    RecurArgs a{};
    a.kind = s.lin_kind;
    a.heads = s.lin_heads;
    a.kv_heads = s.lin_kv_heads;
    a.dim = s.lin_dim;
    a.vdim = s.lin_vdim;
    a.eps = (float)cfg_.rms_norm_eps;
    if (s.lin_kind == LIN_RETENTION) {
        a.q = mix_raw_ + c.lq;
        a.k = mix_raw_ + c.lk;
        a.v = mix_raw_ + c.lv;
        a.gate = mix_raw_ + c.lg;
        a.ldq = a.ldk = a.ldv = a.ld_gate = c.ld;
        a.head_ld = lin_stride(s);
        a.q_scale = 1.0f / std::sqrt((float)s.lin_dim);  // (the keys' factor: the state is linear in them)
        a.decay = w.lin_decay;
    } else {
        const PreparedRows r = prepared_rows(s);
        a.q = lin_rows_ + r.q;
        a.k = lin_rows_ + r.k;
        a.v = lin_rows_ + r.v;
        a.alpha = lin_rows_ + r.alpha;
        a.gate = lin_rows_ + r.gate;
        a.ldq = a.ldk = s.lin_kv_heads * s.lin_dim;
        a.ldv = a.ld_gate = s.lin_heads * s.lin_vdim;
        a.head_ld = s.lin_dim;
        a.q_scale = 1.f;
        a.beta = mix_raw_ + c.lb;
        a.ld_beta = c.ld;
        a.norm_w = w.lin_norm;
    }
    a.state = state_ + w.gla_at;
    a.seq_stride = state_floats_;
    a.row_pos = row_pos;
    a.row_seq = row_seq;
    a.M = M;
    a.runs = pass_runs(M, &a.longest_run);
    a.early = pass_runs_.empty() ? 1 : 0;  // the captured decode step
    a.err_flag = err_flag_;
    a.out = cat_;
    a.ld_out = cat_ld_;
    const bool second = s.mixer == MIX_PARALLEL;  // inputs of the second output projection
    if (!tall) {
        a.out_off = second ? c.k_out : 0;
    } else {
        a.xp = xpack_cat_ + (second ? tc_xpack_bytes(M, c.k_out) : 0);
        a.xp_mpad = tc_mpad(M);
    }
    return a;
}

int Engine::enqueue_sandwich_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int lm_rows, int* launches) {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    const ParallelColumns c = sandwich_columns(s);
    const bool tall = tall_rows(M);
    auto want = [&](int cls) { return only_class_ < 0 || only_class_ == cls; };
    auto prefetch = [&](const LinearW* n) {  // weights of the kernel two launches ahead (streaming passes)
        pf_ptr_ = nullptr;
        pf_bytes_ = 0;
        if (!use_prefetch_ || tall || only_class_ >= 0 || !n || !n->slabs) return;
        pf_ptr_ = n->slabs;
        pf_bytes_ = std::min(n->bytes(), (size_t)24 << 20);
    };
    const LinearW* next_in = l + 1 < L_ ? &layers_[l + 1].in : (lm_rows > 0 ? &lm_head_ : nullptr);
    cudaError_t ce;
    int rc = HM_OK;
    if (l == 0) {
        rc = enqueue_sandwich(M, tall, nullptr, nullptr, w.in_ln, launches);
        if (rc) return rc;
    }
    // what needs no convolution is rotated in the projection's epilogue
    TurnedPairs turn{};
    if (s.mixer == MIX_LINEAR) turn = TurnedPairs{w.turns, lin_stride(s), s.rot.dims, row_pos, 2 * s.lin_heads * lin_stride(s)};
    if (s.mixer == MIX_LATENT) turn = TurnedPairs{w.turns, s.q_stride(), s.rot_dim, row_pos, s.heads * s.q_stride()};
    if (want(PC_QKV)) {
        if (tall) {
            TcArgs a{};
            a.turn = turn;
            if (s.mixer == MIX_LATENT) {  // queries leave as the images the key up-projection reads
                a.split_xp = xpack_q_;
                a.split_n = s.heads * s.q_stride();
                a.split_k = s.q_stride();
                a.split_bytes = tc_xpack_bytes(M, s.q_stride());
            }
            rc = enqueue_tc(w.in, M, xpack_, EPI_STORE, mix_raw_, c.ld, a, launches);
        } else {
            LinOpt o;
            o.turn = turn;
            prefetch(s.mixer == MIX_LATENT ? &w.vup : &w.o);
            rc = enqueue_linear(w.in, M, normed_, H_, PRO_PLAIN, nullptr, EPI_STORE, mix_raw_, c.ld, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    if (want(PC_KV_WRITE) && (s.mixer == MIX_PARALLEL || (s.mixer == MIX_LATENT && s.kv_from < 0))) {
        ce = launch_side(sandwich_side_args(l, M, row_pos, row_seq), sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "side launch");
        ++*launches;
    }
    if (want(PC_RECUR) && s.linear()) {
        ce = launch_recur(recur_args(l, M, tall, row_pos, row_seq), sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "recurrence launch");
        ++*launches;
    }
    if (s.mixer == MIX_PARALLEL && want(PC_ATTN)) {
        GqaAttnArgs a = gqa_attn_args(l, M, tall, row_pos, row_seq);
        a.chunk = s.chunk;
        a.talk = w.talk;
        a.sink = w.sink;
        a.gate = mix_raw_ + c.gate;
        a.ld_gate = c.ld;
        a.gate_kind = s.out_gate;
        a.out = cat_;
        a.ld_out = cat_ld_;
        if (tall) a.xp = xpack_cat_;
        ce = launch_gqa_attn(a, sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "attention launch");
        ++*launches;
    }
    if (s.mixer == MIX_LATENT) {
        const int R = s.latent_rank(), lat = s.heads * R;
        if (want(PC_KUP)) {
            if (tall) {
                TcArgs a{};
                rc = enqueue_tc(w.kup, M, xpack_q_, EPI_STORE, qlat_, lat, a, launches);
            } else {
                LinOpt o;
                o.group_x = s.q_stride();
                prefetch(&w.o);
                rc = enqueue_linear(w.kup, M, mix_raw_ + c.q, c.ld, PRO_PLAIN, nullptr, EPI_STORE, qlat_, lat, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
            }
            if (rc) return rc;
        }
        if (want(PC_ATTN)) {
            rc = enqueue_latent_attn(l, M, tall, row_pos, row_seq, launches);
            if (rc) return rc;
        }
        if (want(PC_VUP)) {
            if (tall) {
                TcArgs a{};
                a.gate = mix_raw_ + c.gate;
                a.ld_gate = c.ld;
                a.gate_per = s.vdim;
                a.xp_out = xpack_cat_;
                rc = enqueue_tc(w.vup, M, xpack_ctx_, EPI_GATE, cat_, cat_ld_, a, launches);
            } else {
                LinOpt o;
                o.group_x = R;
                o.gate = mix_raw_ + c.gate;
                o.ld_gate = c.ld;
                o.gate_per = s.vdim;
                const bool merge = pass_nsplit_ > 1;
                if (merge) o.split = SplitRows{lat_acc_, lat_ml_, pass_nsplit_, s.heads};
                prefetch(s.mlp == MLP_NONE ? next_in : &w.gu);
                rc = enqueue_linear(w.vup, M, ctx_, lat, merge ? PRO_MERGE : PRO_PLAIN, nullptr, EPI_GATE, cat_, cat_ld_, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
            }
            if (rc) return rc;
        }
    }
    const bool both = s.mixer == MIX_PARALLEL;
    const int y_ld = both ? 2 * H_ : H_;
    if (want(PC_O)) {
        if (tall) {
            TcArgs a{};
            rc = enqueue_tc(w.o, M, xpack_cat_, EPI_STORE, sub_, y_ld, a, launches);
        } else {
            LinOpt o;
            o.group_x = both ? c.k_out : 0;
            prefetch(s.mlp == MLP_NONE ? next_in : &w.gu);
            rc = enqueue_linear(w.o, M, cat_, cat_ld_, PRO_PLAIN, nullptr, EPI_STORE, sub_, y_ld, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    // the last norm of a pass is the logits' where every row's are wanted
    const float* after = l + 1 < L_ ? layers_[l + 1].in_ln : final_norm_fits(M, lm_rows) ? final_norm_ : nullptr;
    rc = enqueue_sandwich(M, tall, both ? &w : nullptr, w.norm1b, s.mlp == MLP_NONE ? after : w.post_ln, launches);
    if (rc || s.mlp == MLP_NONE) return rc;
    if (want(PC_GATE_UP)) {
        if (tall) {
            TcArgs a{};
            a.bias = w.gu_bias;
            a.limit = s.limit;
            a.glu_n = s.ff;
            a.xp_out = xpack_act_;
            rc = enqueue_tc(w.gu, M, xpack_, EPI_GLU, act_, s.ff, a, launches);
        } else {
            LinOpt o;
            o.limit = s.limit;
            o.glu_n = s.ff;
            prefetch(next_in);
            rc = enqueue_linear(w.gu, M, normed_, H_, PRO_PLAIN, nullptr, EPI_GLU, act_, s.ff, w.gu_bias, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    if (want(PC_DOWN)) {
        if (tall) {
            TcArgs a{};
            a.bias = w.down_bias;
            rc = enqueue_tc(w.down, M, xpack_act_, EPI_STORE, sub_, H_, a, launches);
        } else {
            prefetch(next_in);
            rc = enqueue_linear(w.down, M, act_, s.ff, PRO_PLAIN, nullptr, EPI_STORE, sub_, H_, w.down_bias, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches);
        }
        if (rc) return rc;
    }
    return enqueue_sandwich(M, tall, nullptr, w.norm2b, after, launches);
}

// Logits of `rows` rows of x; `normed`: the pass's last norm has left them normed.
int Engine::enqueue_sandwich_logits(const float* x, int rows, bool normed, float* dst, const ArgmaxFold& fold, int* launches) {
    const bool tall = tall_rows(rows);
    if (!normed) {
        SandwichArgs a{};
        a.x = const_cast<float*>(x);
        a.next_w = final_norm_;
        a.eps = (float)cfg_.rms_norm_eps;
        a.M = rows;
        a.W = H_;
        a.normed = normed_;
        if (tall) {
            a.xp = xpack_;
            a.xp_mpad = tc_mpad(rows);
        }
        const cudaError_t ce = launch_sandwich(a, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "norm launch");
        ++*launches;
    }
    if (tall) {
        TcArgs a{};
        a.amax_val = amax_val_;
        a.amax_idx = amax_idx_;
        return enqueue_tc(lm_head_, rows, xpack_, EPI_LOGITS, dst, V_, a, launches);
    }
    return enqueue_linear(lm_head_, rows, normed_, H_, PRO_PLAIN, nullptr, EPI_LOGITS, dst, V_, nullptr, nullptr, -1, nullptr, nullptr, amax_val_, amax_idx_, launches, &fold);
}

}  // namespace hm
