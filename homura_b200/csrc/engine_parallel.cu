// Engine parts for listed designs whose mixer and feed-forward read one norm of the residual and are added to it together: weights,
// scratch, and the launches of one layer.  Beside engine_listed.cu and engine_gqa.cu, whose attention and experts they use.
//
// Everything that reads the norm is one projection (ParallelColumns), and so is everything that joins the residual:
//   in      queries, keys, values, gates, latents, router logits, gate and up of the dense or shared feed-forward
//   side    convolutions, rotations, page slots; gated linear attention; activations; the router's choice          (side.cu)
//   attn    softmax attention with its output gate
//   out     residual += [attention | linear attention | feed-forward] projected
//   experts gate and up, down, residual
// Latent attention has, between side and out: the queries out of their latent (rotated in the epilogue), key up, attention, value up.
// With many rows the norm is a launch in front of `in`, which also adds up the experts' partial results (sum_norm).
#include "engine_parallel.h"

#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <cstring>

#include "engine_util.h"
#include "gemm_tc.h"

namespace hm {

ParallelColumns parallel_columns(const LayerSpec& s) {
    ParallelColumns c;
    int at = 0;
    auto take = [&](int n) {
        const int first = at;
        at += (n + 7) / 8 * 8;
        return first;
    };
    if (s.paged_kv()) {
        c.q = take(s.heads * s.dim + s.kv_heads * (s.dim + s.vdim));
        c.k = c.q + s.heads * s.dim;
        c.v = c.k + s.kv_heads * s.dim;
        c.gates = s.out_gate == GATE_ELEM ? s.heads * s.vdim : s.out_gate == GATE_HEAD ? s.heads : 0;
        c.gate = take(c.gates);
    } else {
        c.dq = take(s.q_rank);
        c.dkv = take(s.latent_rank());
    }
    if (s.mixer == MIX_PARALLEL) {
        c.lq = take(s.lin_heads * s.lin_dim);
        c.lk = take(s.lin_heads * s.lin_dim);
        c.lv = take(s.lin_heads * s.lin_vdim);
        c.lg = take(s.lin_heads * s.lin_vdim);
        c.la = take(s.decay_rank);
    }
    if (s.mlp == MLP_MOE) {
        c.router = take(s.experts);
        if (s.shared_ff) c.row_gate = take(1);
    }
    c.ff = s.mlp == MLP_GLU ? s.ff : s.mlp == MLP_MOE ? s.shared_ff : 0;
    c.ff_gate = take(c.ff);
    c.ff_up = take(c.ff);
    c.n = c.ld = at;
    auto input = [&](int n) {
        const int first = c.k_out;
        c.k_out += (n + 63) / 64 * 64;
        return first;
    };
    c.vals = input(s.heads * s.vdim);
    if (s.mixer == MIX_PARALLEL) c.lin_in = input(s.lin_heads * s.lin_vdim);
    c.ff_in = input(c.ff);
    return c;
}

// ---- weights -------------------------------------------------------------------------------------

void Engine::note_shape(const std::string& name, const std::vector<int64_t>& shape) {
    if (!(spec_.parallel || spec_.sandwich) || name.empty() || name[0] != 'l' || shape.size() != 2 || shape[0] < 1 || shape[0] > 1 << 16) return;
    const size_t dot = name.find('.');
    if (dot == std::string::npos || name.find_first_not_of("0123456789", 1) != dot) return;
    const long l = std::atol(name.c_str() + 1);
    if (l < 0 || l >= L_) return;
    LayerSpec& s = spec_.layers[l];
    if (name.substr(dot) == ".mix.right.a1" && s.decay_rank == 0) s.decay_rank = (int)shape[0];
    if (name.substr(dot) == ".mix.right.g1" && s.lin_kind == LIN_DELTA && s.gate_rank == 0) s.gate_rank = (int)shape[0];
}

int Engine::upload(float** dst, const std::vector<float>& v) {
    HM_CUDA(cudaMalloc(dst, v.size() * 4));
    HM_CUDA(cudaMemcpy(*dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
    return HM_OK;
}

int Engine::load_bigram(int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    if (ndim != 2 || shape[0] != spec_.bigram_buckets + 1 || shape[1] != H_) return fail(HM_ERR_INVALID, "unexpected shape for tensor bigram");
    if (dtype != HM_BF16 || nbytes != (size_t)shape[0] * H_ * 2) return fail(HM_ERR_UNSUPPORTED, "the bigram embedding must be stored as bf16");
    if (bigram_) return fail(HM_ERR_STATE, "tensor loaded twice: bigram");
    const int rc = stage(host, nbytes, reinterpret_cast<void**>(&bigram_));
    if (rc) return rc;
    HM_CUDA(cudaStreamSynchronize(stream_));
    return HM_OK;
}

// Inputs [k_off, k_off + k_part) of a projection over k_total inputs whose input parts come as tensors of their own.
int Engine::load_inputs(LinearW& L, int k_total, int k_off, int k_part, int N, int dtype, const void* host, size_t nbytes) {
    if (dtype != HM_BF16) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
    if (nbytes != (size_t)N * k_part * 2) return fail(HM_ERR_INVALID, "tensor byte size does not match its shape");
    L.K = k_total;
    L.N = N;
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
    cudaError_t ce = room(&L.slabs, (size_t)((N + SLAB - 1) / SLAB) * k_total * SLAB * 2);
    if (ce == cudaSuccess) ce = launch_pack_slabs_from_nk((const uint16_t*)tmp, N, k_part, L.slabs, 0, -1, stream_, k_total, k_off);
    if (use_tc_) {
        if (ce == cudaSuccess) ce = room(&L.tc, tc_packed_elems(k_total, N) * 2);
        if (ce == cudaSuccess) ce = launch_pack_tc((const uint16_t*)tmp, N, k_part, false, L.tc, 0, -1, stream_, k_total, k_off);
    }
    if (ce == cudaSuccess) ce = cudaStreamSynchronize(stream_);
    cudaFree(tmp);
    if (ce != cudaSuccess) return cuda_fail(ce, "load_inputs");
    L.loaded_parts++;
    return HM_OK;
}

// Keys are W_uk c, so a query meets the latents as W_uk^T q; its rotated part passes to the end of the cached row.
int Engine::load_key_up(LayerW& w, const LayerSpec& s, const std::string& name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    const int R = s.latent_rank(), qs = s.q_stride();
    const uint16_t* bits = static_cast<const uint16_t*>(host);
    if (ndim != 2 || shape[0] != (int64_t)s.heads * s.dim || shape[1] != s.kv_rank) return fail(HM_ERR_INVALID, "unexpected shape for tensor " + name);
    if (dtype != HM_BF16 || nbytes != (size_t)s.heads * s.dim * s.kv_rank * 2) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
    std::vector<uint16_t> m((size_t)s.heads * qs * R, 0);
    for (int h = 0; h < s.heads; ++h) {
        uint16_t* g = &m[(size_t)h * qs * R];
        for (int e = 0; e < s.rot_dim; ++e) g[(size_t)e * R + s.kv_rank + e] = 0x3f80;  // 1
        for (int d = 0; d < s.dim; ++d) std::memcpy(g + (size_t)(s.rot_dim + d) * R, bits + ((size_t)h * s.dim + d) * s.kv_rank, (size_t)s.kv_rank * 2);
    }
    return load_grouped(w.kup, s.heads, qs, R, true, dtype, m.data(), m.size() * 2);
}

// The rotated part of a cached row is no value.
int Engine::load_value_up(LayerW& w, const LayerSpec& s, const std::string& name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    const int R = s.latent_rank();
    const uint16_t* bits = static_cast<const uint16_t*>(host);
    if (ndim != 2 || shape[0] != (int64_t)s.heads * s.vdim || shape[1] != s.kv_rank) return fail(HM_ERR_INVALID, "unexpected shape for tensor " + name);
    if (dtype != HM_BF16 || nbytes != (size_t)s.heads * s.vdim * s.kv_rank * 2) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
    std::vector<uint16_t> m((size_t)s.heads * s.vdim * R, 0);
    for (int i = 0; i < s.heads * s.vdim; ++i) std::memcpy(&m[(size_t)i * R], bits + (size_t)i * s.kv_rank, (size_t)s.kv_rank * 2);
    return load_grouped(w.vup, s.heads, R, s.vdim, false, dtype, m.data(), m.size() * 2);
}

int Engine::load_parallel_tensor(int layer, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    LayerW& w = layers_[layer];
    LayerSpec& s = spec_.layers[layer];
    size_t n = 1;
    for (int i = 0; i < ndim; ++i) n *= (size_t)shape[i];
    auto bad_shape = [&]() { return fail(HM_ERR_INVALID, "unexpected shape for tensor " + name); };
    auto is2 = [&](int64_t a, int64_t b) { return ndim == 2 && shape[0] == a && shape[1] == b; };
    auto unknown = [&]() { return fail(HM_ERR_INVALID, "unknown tensor name: " + name); };
    if (s.mlp == MLP_MOE) {
        int rc = HM_OK;
        if (load_expert_tensor(w, s, name, rest, dtype, shape, ndim, host, nbytes, &rc)) return rc;
    }
    if (std::find(w.seen.begin(), w.seen.end(), rest) != w.seen.end()) return fail(HM_ERR_STATE, "tensor loaded twice: " + name);
    if (s.mixer == MIX_PARALLEL && s.decay_rank == 0) {
        if (rest == "mix.right.a1" && ndim == 2) note_shape(name, {shape[0], shape[1]});
        else return fail(HM_ERR_STATE, "mix.right.a1 must be loaded before the other tensors of its layer (hm_model_load does so)");
    }
    const ParallelColumns c = parallel_columns(s);
    // parts of the input projection, vectors, inputs of the output projection
    auto in = [&](int off, int part) { return is2(part, H_) ? load_linear(w.in, H_, c.n, off, part, -1, dtype, host, nbytes) : bad_shape(); };
    auto vec = [&](float** dst, size_t total, size_t off, size_t len, bool flat = true) { return n != len || (flat && ndim != 1) ? bad_shape() : load_vec_f32(dst, total, off, dtype, host, n, nbytes); };
    auto out = [&](int off, int part) { return is2(H_, part) ? load_inputs(w.o, c.k_out, off, part, H_, dtype, host, nbytes) : bad_shape(); };
    const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim, channels = nq + nk + nv;
    const int lk = s.lin_heads * s.lin_dim, lv = s.lin_heads * s.lin_vdim;
    auto attention = [&](const std::string& t) -> int {
        const struct { const char* name; int off, len; } qkv[3] = {{"q", 0, nq}, {"k", nq, nk}, {"v", nq + nk, nv}};
        for (auto& p : qkv) {
            if (t == p.name) return in(c.q + p.off, p.len);
            if (s.qkv_bias && t == std::string(p.name) + ".b") return vec(&w.in_bias, c.n, c.q + p.off, p.len);
            if (s.conv > 0 && t == std::string(p.name) + ".conv") return is2(p.len, s.conv) ? vec(&w.conv_w, (size_t)channels * s.conv, (size_t)p.off * s.conv, n, false) : bad_shape();
        }
        if (t == "sink" && s.sink) return vec(&w.sink, s.heads, 0, s.heads);
        if (t == "g" && c.gates) return in(c.gate, c.gates);
        if (t == "o") return out(c.vals, s.heads * s.vdim);
        return unknown();
    };
    auto to_f32 = [&](size_t i) {
        if (dtype == HM_F32) return static_cast<const float*>(host)[i];
        const uint32_t u = (uint32_t)static_cast<const uint16_t*>(host)[i] << 16;
        float f;
        std::memcpy(&f, &u, 4);
        return f;
    };
    auto linear = [&](const std::string& t) -> int {
        if (t == "q") return in(c.lq, lk);
        if (t == "k") return in(c.lk, lk);
        if (t == "v") return in(c.lv, lv);
        if (t == "g") return in(c.lg, lv);
        if (t == "a1") return in(c.la, s.decay_rank);
        if (t == "o") return out(c.lin_in, lv);
        if (t == "norm") return vec(&w.lin_norm, s.lin_vdim, 0, s.lin_vdim);
        if (t == "a2.b") return vec(&w.lin_bias, lk, 0, lk);
        if (t != "a2") return unknown();
        if (!is2(lk, s.decay_rank)) return bad_shape();
        if ((dtype != HM_BF16 && dtype != HM_F32) || nbytes != n * (dtype == HM_BF16 ? 2 : 4)) return fail(HM_ERR_UNSUPPORTED, "decay projections must be stored as bf16 or f32");
        std::vector<float> up(n);  // [heads][rank][dim]
        for (int h = 0; h < s.lin_heads; ++h)
            for (int d = 0; d < s.lin_dim; ++d)
                for (int r = 0; r < s.decay_rank; ++r) up[((size_t)h * s.decay_rank + r) * s.lin_dim + d] = to_f32(((size_t)h * s.lin_dim + d) * s.decay_rank + r);
        return upload(&w.lin_up, up);
    };
    const uint16_t* bits = static_cast<const uint16_t*>(host);
    auto bf16 = [&]() { return dtype == HM_BF16 && nbytes == n * 2; };
    auto latent = [&](const std::string& t) -> int {
        const int R = s.latent_rank(), qs = s.q_stride(), half = s.rot_dim / 2;
        if (t == "dq") return in(c.dq, s.q_rank);
        if (t == "dkv") return in(c.dkv, R);
        if (t == "dq.norm") return vec(&w.q_norm, s.q_rank, 0, s.q_rank);
        if (t == "dkv.norm") return vec(&w.latent_norm, s.kv_rank, 0, s.kv_rank);
        if (t == "o") return out(c.vals, s.heads * s.vdim);
        if (t == "uq") {
            // a head's rows: the rotated pairs side by side, the unrotated ones, padding to q_stride
            const int per = s.dim + s.rot_dim;
            if (!is2((int64_t)s.heads * per, s.q_rank)) return bad_shape();
            if (!bf16()) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
            std::vector<uint16_t> m((size_t)s.heads * qs * s.q_rank, 0);
            for (int h = 0; h < s.heads; ++h)
                for (int e = 0; e < per; ++e) {
                    const int r = e - s.dim, row = r < 0 ? s.rot_dim + e : r < half ? 2 * r : 2 * (r - half) + 1;
                    std::memcpy(&m[((size_t)h * qs + row) * s.q_rank], bits + ((size_t)h * per + e) * s.q_rank, (size_t)s.q_rank * 2);
                }
            return load_linear(w.uq, s.q_rank, s.heads * qs, 0, s.heads * qs, -1, dtype, m.data(), m.size() * 2);
        }
        if (t == "uk") return load_key_up(w, s, name, dtype, shape, ndim, host, nbytes);
        if (t == "uv") return load_value_up(w, s, name, dtype, shape, ndim, host, nbytes);
        return unknown();
    };
    auto feed_forward = [&](const std::string& t) -> int {
        std::string part = t;
        if (s.mlp == MLP_MOE) {
            if (t == "router") return in(c.router, s.experts);
            if (t.compare(0, 7, "shared.") != 0 || !c.ff) return unknown();
            part = t.substr(7);
            if (part == "sg") return in(c.row_gate, 1);
        } else if (s.mlp != MLP_GLU) {
            return unknown();
        }
        if (part == "gate") return in(c.ff_gate, c.ff);
        if (part == "up") return in(c.ff_up, c.ff);
        if (part == "down") return out(c.ff_in, c.ff);
        return unknown();
    };
    int rc;
    if (rest.compare(0, 4, "mlp.") == 0) rc = feed_forward(rest.substr(4));
    else if (s.mixer == MIX_PARALLEL && rest.compare(0, 9, "mix.left.") == 0) rc = attention(rest.substr(9));
    else if (s.mixer == MIX_PARALLEL && rest.compare(0, 10, "mix.right.") == 0) rc = linear(rest.substr(10));
    else if (s.mixer == MIX_GQA && rest.compare(0, 4, "mix.") == 0) rc = attention(rest.substr(4));
    else if (s.mixer == MIX_LATENT && rest.compare(0, 4, "mix.") == 0) rc = latent(rest.substr(4));
    else rc = unknown();
    if (rc == HM_OK) w.seen.push_back(rest);
    return rc;
}

int Engine::finalize_parallel() {
    if (spec_.bigram_buckets > 0 && !bigram_) return fail(HM_ERR_STATE, "missing weight: bigram");
    for (int l = 0; l < L_; ++l) {
        LayerW& w = layers_[l];
        const LayerSpec& s = spec_.layers[l];
        std::vector<std::string> need;
        auto attention = [&](const std::string& p) {
            for (const char* t : {"q", "k", "v"}) {
                need.push_back(p + t);
                if (s.qkv_bias) need.push_back(p + t + ".b");
                if (s.conv > 0) need.push_back(p + t + ".conv");
            }
            if (s.sink) need.push_back(p + "sink");
            if (s.out_gate != GATE_NONE) need.push_back(p + "g");
            need.push_back(p + "o");
        };
        if (s.mixer == MIX_GQA) attention("mix.");
        if (s.mixer == MIX_PARALLEL) {
            attention("mix.left.");
            for (const char* t : {"q", "k", "v", "g", "o", "norm", "a1", "a2", "a2.b"}) need.push_back(std::string("mix.right.") + t);
        }
        if (s.mixer == MIX_LATENT)
            for (const char* t : {"dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o"}) need.push_back(std::string("mix.") + t);
        if (s.mlp == MLP_GLU)
            for (const char* t : {"gate", "up", "down"}) need.push_back(std::string("mlp.") + t);
        if (s.mlp == MLP_MOE) {
            need.push_back("mlp.router");
            if (s.shared_ff)
                for (const char* t : {"gate", "up", "down", "sg"}) need.push_back(std::string("mlp.shared.") + t);
        }
        const std::string at = "missing weight in layer " + std::to_string(l) + ": ";
        if (!w.in_ln) return fail(HM_ERR_STATE, at + "norm1");
        for (const std::string& t : need)
            if (std::find(w.seen.begin(), w.seen.end(), t) == w.seen.end()) return fail(HM_ERR_STATE, at + t);
        for (int e = 0; e < (s.mlp == MLP_MOE ? s.experts : 0); ++e)
            if ((size_t)e >= w.exp_seen.size() || w.exp_seen[e] != 7) return fail(HM_ERR_STATE, at + "mlp.e" + std::to_string(e));
        if (s.rot.dims) {
            const std::vector<double> t = rotation_turns(s.rot);
            HM_CUDA(cudaMalloc(&w.turns, t.size() * 8));
            HM_CUDA(cudaMemcpy(w.turns, t.data(), t.size() * 8, cudaMemcpyHostToDevice));
        }
    }
    return HM_OK;
}

// ---- scratch ---------------------------------------------------------------------------------------

void Engine::free_parallel_scratch() {
    auto fr = [](auto*& p) {
        if (p) cudaFree(p);
        p = nullptr;
    };
    fr(normed_); fr(cat_); fr(xpack_cat_); fr(xpack_cq_); fr(lin_rows_);
}

int Engine::alloc_parallel_scratch() {
    if (!spec_.parallel) return HM_OK;
    int k_out = 1, q_rank = 1;
    for (const LayerSpec& s : spec_.layers) {
        k_out = std::max(k_out, parallel_columns(s).k_out);
        q_rank = std::max(q_rank, s.q_rank);
    }
    auto get = [&](auto** p, size_t count) -> cudaError_t {
        const cudaError_t e = cudaMalloc((void**)p, count * sizeof(**p));
        return e == cudaSuccess ? cudaMemset(*p, 0, count * sizeof(**p)) : e;
    };
    cat_ld_ = k_out;
    HM_CUDA(get(&normed_, (size_t)TC_ROWS * H_));
    HM_CUDA(get(&cat_, (size_t)TC_ROWS * k_out));
    if (use_tc_) {
        HM_CUDA(get(&xpack_cat_, tc_xpack_bytes(TC_ROWS, k_out)));
        HM_CUDA(get(&xpack_cq_, tc_xpack_bytes(TC_ROWS, q_rank)));
    }
    return HM_OK;
}

// ---- one layer ---------------------------------------------------------------------------------------

SideArgs Engine::side_args(int l, int M, bool tall, const ParallelColumns& c, const int32_t* row_pos, const int32_t* row_seq) const {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    SideArgs a{};
    a.M = M;
    a.ld = c.ld;
    a.xp_mpad = tc_mpad(M);
    a.eps = (float)cfg_.rms_norm_eps;
    a.row_pos = row_pos;
    a.row_seq = row_seq;
    int longest = 1;
    const GqaRuns runs = pass_runs(M, &longest);
    if (s.paged_kv()) {
        a.has_post = 1;
        GqaPostArgs& p = a.post;
        p.pool = gqa_pool(l);
        p.raw = mix_raw_ + c.q;
        p.ld = c.ld;
        p.M = M;
        p.heads = s.heads;
        p.qk_norm = s.qk_norm;
        p.eps = a.eps;
        p.q_scale = (float)(s.scale * 1.4426950408889634);
        p.row_pos = row_pos;
        p.row_seq = row_seq;
        p.q_out = q_;
        p.taps = s.conv;
        p.conv_w = w.conv_w;
        p.conv_state = state_ ? state_ + w.conv_at : nullptr;
        p.conv_stride = state_floats_;
        p.runs = runs;
        p.rot_dims = s.rot.dims;
        p.turns = w.turns;
    } else {
        a.has_latent = 1;
        LatentSide& t = a.latent;
        t.pool = latent_pool(l);
        t.c = mix_raw_ + c.dkv;
        t.w = w.latent_norm;
        t.rot_pairs = s.rot_dim / 2;
        t.turns = w.turns;
        t.cq = mix_raw_ + c.dq;
        t.q_rank = s.q_rank;
        t.q_w = w.q_norm;
        t.q_xp = tall ? xpack_cq_ : nullptr;
    }
    if (s.mixer == MIX_PARALLEL) {
        a.has_gla = 1;
        GlaArgs& g = a.gla;
        g.heads = s.lin_heads;
        g.dim = s.lin_dim;
        g.vdim = s.lin_vdim;
        g.rank = s.decay_rank;
        g.raw = mix_raw_;
        g.ld = c.ld;
        g.q_off = c.lq;
        g.k_off = c.lk;
        g.v_off = c.lv;
        g.g_off = c.lg;
        g.a_off = c.la;
        g.q_scale = 1.0f / std::sqrt((float)s.lin_dim);
        g.up = w.lin_up;
        g.bias = w.lin_bias;
        g.inv_tau = 1.0f / s.lin_tau;
        g.norm_w = w.lin_norm;
        g.eps = a.eps;
        g.out_scale = s.right_scale;
        g.state = state_ + w.gla_at;
        g.seq_stride = state_floats_;
        g.row_pos = row_pos;
        g.row_seq = row_seq;
        g.M = M;
        g.runs = runs;
        g.longest_run = longest;
        g.err_flag = err_flag_;
        g.early = pass_runs_.empty() ? 1 : 0;  // the captured decode step
        g.out = cat_;
        g.ld_out = cat_ld_;
        g.out_off = c.lin_in;
        g.xp = tall ? xpack_cat_ : nullptr;
        g.xp_mpad = a.xp_mpad;
    }
    MlpSide& f = a.mlp;
    f.ff = c.ff;
    f.act = s.act;
    f.gate = mix_raw_ + c.ff_gate;
    f.up = mix_raw_ + c.ff_up;
    f.out = cat_;
    f.ld_out = cat_ld_;
    f.out_off = c.ff_in;
    f.xp = tall ? xpack_cat_ : nullptr;
    if (s.mlp == MLP_MOE) {
        if (c.ff) f.row_gate = mix_raw_ + c.row_gate;
        f.logits = mix_raw_ + c.router;
        f.route = RouteSpec{nullptr, s.experts, s.experts, s.top, s.router_scale, route_out(tall)};
        if (!tall) {
            f.x = h_;
            f.W = H_;
            f.w = w.in_ln;
            f.normed = normed_;
        }
    }
    return a;
}

int Engine::enqueue_parallel_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int next_lm_rows, int* launches) {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    const ParallelColumns c = parallel_columns(s);
    const bool tall = tall_rows(M), moe = s.mlp == MLP_MOE;
    auto want = [&](int cls) { return only_class_ < 0 || only_class_ == cls; };
    auto prefetch = [&](const LinearW* n) {  // weights of the kernel two launches ahead (streaming passes)
        pf_ptr_ = nullptr;
        pf_bytes_ = 0;
        if (!use_prefetch_ || tall || only_class_ >= 0 || !n || !n->slabs) return;
        pf_ptr_ = n->slabs;
        pf_bytes_ = std::min(n->bytes(), (size_t)24 << 20);
    };
    const LinearW* next_in = l + 1 < L_ ? &layers_[l + 1].in : (next_lm_rows > 0 ? &lm_head_ : nullptr);
    // residual + parts, and its norm for the projection behind
    auto sum_norm = [&](int parts, const float* norm_w) -> int {
        if (!want(PC_NORM) || (!parts && !norm_w)) return HM_OK;
        SumNormArgs a{};
        a.x = h_;
        a.y = sub_;
        a.parts = parts;
        a.part_stride = (size_t)TC_ROWS * H_;
        a.M = M;
        a.W = H_;
        a.w = norm_w;
        a.eps = (float)cfg_.rms_norm_eps;
        a.xp = xpack_;
        a.xp_mpad = tc_mpad(M);
        const cudaError_t e = launch_sum_norm(a, stream_, pdl_);
        if (e != cudaSuccess) return cuda_fail(e, "norm and pack launch");
        ++*launches;
        return HM_OK;
    };
    cudaError_t ce;
    int rc = HM_OK;
    if (tall && l == 0) {  // later layers find the image where the layer in front left it
        rc = sum_norm(0, w.in_ln);
        if (rc) return rc;
    }
    if (want(PC_QKV)) {
        if (tall) {
            TcArgs a{};
            a.bias = w.in_bias;
            rc = enqueue_tc(w.in, M, xpack_, EPI_STORE, mix_raw_, c.ld, a, launches);
        } else {
            prefetch(s.mixer == MIX_LATENT ? &w.uq : &w.o);
            rc = enqueue_linear(w.in, M, h_, H_, PRO_RMSNORM, w.in_ln, EPI_STORE, mix_raw_, c.ld, w.in_bias, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches);
        }
        if (rc) return rc;
    }
    if (want(PC_KV_WRITE)) {
        ce = launch_side(side_args(l, M, tall, c, row_pos, row_seq), sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "side launch");
        ++*launches;
        if (experts_seen_ && moe) {
            rc = count_experts(M, s);
            if (rc) return rc;
        }
    }
    if (s.paged_kv()) {
        if (want(PC_ATTN)) {
            GqaAttnArgs a = gqa_attn_args(l, M, tall, row_pos, row_seq);
            a.window = s.window;
            a.keep_first = s.keep_first;
            a.sink = w.sink;
            a.gate = mix_raw_ + c.gate;
            a.ld_gate = c.ld;
            a.gate_kind = s.out_gate;
            a.out_scale = s.mixer == MIX_PARALLEL ? s.left_scale : 0.f;
            a.out = cat_;
            a.ld_out = cat_ld_;
            a.out_off = c.vals;
            if (tall) a.xp = xpack_cat_;
            ce = launch_gqa_attn(a, sm_count_, stream_, pdl_);
            if (ce != cudaSuccess) return cuda_fail(ce, "attention launch");
            ++*launches;
        }
    } else {
        const int R = s.latent_rank(), lat = s.heads * R, qs = s.q_stride(), qn = s.heads * qs;
        const TurnedPairs turn{w.turns, qs, s.rot_dim, row_pos};
        if (want(PC_QUP)) {
            if (tall) {
                TcArgs a{};
                a.turn = turn;
                a.split_xp = xpack_q_;  // queries leave as the images the next projection reads
                a.split_n = qn;
                a.split_k = qs;
                a.split_bytes = tc_xpack_bytes(M, qs);
                rc = enqueue_tc(w.uq, M, xpack_cq_, EPI_STORE, q_, qn, a, launches);
            } else {
                LinOpt o;
                o.turn = turn;
                prefetch(&w.vup);
                rc = enqueue_linear(w.uq, M, mix_raw_ + c.dq, c.ld, PRO_RMSNORM, w.q_norm, EPI_STORE, q_, qn, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
            }
            if (rc) return rc;
        }
        if (want(PC_KUP)) {
            if (tall) {
                TcArgs a{};
                rc = enqueue_tc(w.kup, M, xpack_q_, EPI_STORE, qlat_, lat, a, launches);
            } else {
                LinOpt o;
                o.group_x = qs;
                prefetch(&w.o);
                rc = enqueue_linear(w.kup, M, q_, qn, PRO_PLAIN, nullptr, EPI_STORE, qlat_, lat, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
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
                a.split_xp = xpack_cat_;
                a.split_n = s.heads * s.vdim;
                a.split_k = 1 << 30;  // one image
                rc = enqueue_tc(w.vup, M, xpack_ctx_, EPI_STORE, cat_, cat_ld_, a, launches);
            } else {
                LinOpt o;
                o.group_x = R;
                const bool merge = pass_nsplit_ > 1;
                if (merge) o.split = SplitRows{lat_acc_, lat_ml_, pass_nsplit_, s.heads};
                prefetch(next_in);
                rc = enqueue_linear(w.vup, M, ctx_, lat, merge ? PRO_MERGE : PRO_PLAIN, nullptr, EPI_STORE, cat_, cat_ld_, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
            }
            if (rc) return rc;
        }
    }
    if (want(PC_O)) {
        if (tall) {
            TcArgs a{};
            a.resid = h_;
            rc = enqueue_tc(w.o, M, xpack_cat_, EPI_STORE, h_, H_, a, launches);
        } else {
            prefetch(next_in);
            rc = enqueue_linear(w.o, M, cat_, cat_ld_, PRO_PLAIN, nullptr, EPI_STORE, h_, H_, nullptr, h_, l, row_pos, row_seq, nullptr, nullptr, launches);
        }
        if (rc) return rc;
    }
    int parts = 0;
    if (moe) {
        rc = enqueue_experts(l, M, tall, normed_, h_, tall ? sub_ : h_, &parts, launches);
        if (rc) return rc;
    }
    return tall ? sum_norm(moe ? parts : 0, l + 1 < L_ ? layers_[l + 1].in_ln : nullptr) : HM_OK;
}

}  // namespace hm
