// Engine parts for listed designs with grouped-query attention whose sublayers read the residual itself and normalise what they
// give back: weights, scratch, and the launches of one layer.  Beside engine_listed.cu, which holds what all listed designs share.
//
// A layer with a mixture of experts is, per pass,
//   in      [queries | keys | values]  <- residual
//   post    query and key norms, temperature, blended values; page slots            (gqa_attn.cu)
//   attn    softmax attention with distance biases                                  (gqa_attn.cu)
//   o       output projection
//   norm    residual += mult * norm(o); router over the new residual                (moe.cu)
//   experts gate and up, down
//   norm    residual += mult * norm(experts + identity)
#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <cstring>

#include "engine.h"
#include "engine_util.h"
#include "gemm_tc.h"

namespace hm {

namespace {
int qkv_cols(const LayerSpec& s) { return s.heads * s.dim + s.kv_heads * (s.dim + s.vdim); }
int qkv_ld(const LayerSpec& s) { return (qkv_cols(s) + 3) / 4 * 4; }

// Row of the bias table for a key n tokens back: a row per distance below half the table, then logarithmic steps up to `reach`.
int distance_row(int n, int rows, double reach) {
    const int half = rows / 2;
    if (n < half) return n;
    if (n >= reach || reach <= half || half == 0) return rows - 1;
    // (a distance that lies exactly on a step belongs to the step's upper side)
    const int r = half + (int)std::floor(std::log((double)n / half) / std::log(reach / half) * (rows - half) + 1e-9);
    return std::min(rows - 1, r);
}
}  // namespace

// ---- weights -------------------------------------------------------------------------------------

// [rows, heads] by bucket -> [heads][reach + 1] by distance, in units of the base-2 exponent.
int Engine::load_bias_table(LayerW& w, const LayerSpec& s, int dtype, const int64_t* shape, const void* host, size_t nbytes) {
    const int rows = (int)shape[0];
    const size_t n = (size_t)rows * s.heads;
    if ((dtype != HM_BF16 && dtype != HM_F32) || nbytes != n * (dtype == HM_BF16 ? 2 : 4)) return fail(HM_ERR_UNSUPPORTED, "distance biases must be stored as bf16 or f32");
    auto at = [&](int r, int h) {
        const size_t i = (size_t)r * s.heads + h;
        if (dtype == HM_F32) return static_cast<const float*>(host)[i];
        const uint32_t u = (uint32_t)static_cast<const uint16_t*>(host)[i] << 16;
        float f;
        std::memcpy(&f, &u, 4);
        return f;
    };
    w.reach = std::max((int)std::ceil(s.bias_reach), rows / 2);
    std::vector<float> t((size_t)s.heads * (w.reach + 1));
    for (int d = 0; d <= w.reach; ++d) {
        const int r = distance_row(d, rows, s.bias_reach);
        for (int h = 0; h < s.heads; ++h) t[(size_t)h * (w.reach + 1) + d] = (float)(at(r, h) * 1.4426950408889634);
    }
    HM_CUDA(cudaMalloc(&w.rel, t.size() * 4));
    HM_CUDA(cudaMemcpy(w.rel, t.data(), t.size() * 4, cudaMemcpyHostToDevice));
    return HM_OK;
}

// part 0 = gate, 1 = up, 2 = down
int Engine::load_expert(LayerW& w, const LayerSpec& s, int expert, int part, int dtype, const void* host, size_t nbytes) {
    if (dtype != HM_BF16) return fail(HM_ERR_UNSUPPORTED, "experts of this design must be stored as bf16");
    if (nbytes != (size_t)s.ff * H_ * 2) return fail(HM_ERR_INVALID, "tensor byte size does not match its shape");
    const size_t gu = expert_gu_elems(H_, s.ff), down = expert_down_elems(H_, s.ff);
    auto room = [&](uint16_t** p, size_t elems) -> cudaError_t {
        if (*p) return cudaSuccess;
        const cudaError_t e = cudaMalloc(p, elems * 2);
        return e == cudaSuccess ? cudaMemsetAsync(*p, 0, elems * 2, stream_) : e;
    };
    cudaError_t ce = part < 2 ? room(&w.exp_gu, s.experts * gu) : room(&w.exp_down, s.experts * down);
    if (ce != cudaSuccess) return cuda_fail(ce, "experts");
    void* tmp = nullptr;
    const int rc = stage(host, nbytes, &tmp);
    if (rc) return rc;
    const uint16_t* src = static_cast<const uint16_t*>(tmp);
    ce = part < 2 ? launch_pack_tc(src, s.ff, H_, false, w.exp_gu + expert * gu, 0, part, stream_) : launch_pack_tc(src, H_, s.ff, false, w.exp_down + expert * down, 0, -1, stream_);
    if (ce == cudaSuccess) ce = cudaStreamSynchronize(stream_);
    cudaFree(tmp);
    if (ce != cudaSuccess) return cuda_fail(ce, "load_expert");
    w.exp_seen.resize(s.experts, 0);
    w.exp_seen[expert] |= (uint8_t)(1 << part);
    cfg_.weight_dtype = HM_BF16;
    return HM_OK;
}

// mlp.e<index>.gate / up / down; false: another tensor
bool Engine::load_expert_tensor(LayerW& w, const LayerSpec& s, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes, int* rc) {
    const size_t dot = rest.find('.', 5);
    if (rest.compare(0, 5, "mlp.e") != 0 || dot == std::string::npos || dot <= 5 || rest.find_first_not_of("0123456789", 5) != dot) return false;
    const long e = std::atol(rest.c_str() + 5);
    const std::string what = rest.substr(dot + 1);
    const int part = what == "gate" ? 0 : what == "up" ? 1 : what == "down" ? 2 : -1;
    if (part < 0) return false;
    if (e >= s.experts) *rc = fail(HM_ERR_INVALID, "expert index out of range in " + name);
    else if (ndim != 2 || shape[0] != (part < 2 ? s.ff : H_) || shape[1] != (part < 2 ? H_ : s.ff)) *rc = fail(HM_ERR_INVALID, "unexpected shape for tensor " + name);
    else if ((size_t)e < w.exp_seen.size() && (w.exp_seen[e] >> part & 1)) *rc = fail(HM_ERR_STATE, "tensor loaded twice: " + name);
    else *rc = load_expert(w, s, (int)e, part, dtype, host, nbytes);
    return true;
}

int Engine::load_gqa_tensor(LayerW& w, const LayerSpec& s, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    size_t n = 1;
    for (int i = 0; i < ndim; ++i) n *= (size_t)shape[i];
    auto is2 = [&](int64_t a, int64_t b) { return ndim == 2 && shape[0] == a && shape[1] == b; };
    auto bad_shape = [&]() { return fail(HM_ERR_INVALID, "unexpected shape for tensor " + name); };
    auto twice = [&]() { return fail(HM_ERR_STATE, "tensor loaded twice: " + name); };
    auto vec = [&](float** dst, int len) {
        if (n != (size_t)len || ndim > 1) return bad_shape();
        return *dst ? twice() : load_vec_f32(dst, len, 0, dtype, host, n, nbytes);
    };
    auto lin = [&](LinearW& L, int K, int total, int off, int part) { return is2(part, K) ? load_linear(L, K, total, off, part, -1, dtype, host, nbytes) : bad_shape(); };
    const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
    if (rest == "mix.q") return lin(w.in, H_, qkv_cols(s), 0, nq);
    if (rest == "mix.k") return lin(w.in, H_, qkv_cols(s), nq, nk);
    if (rest == "mix.v") return lin(w.in, H_, qkv_cols(s), nq + nk, nv);
    if (rest == "mix.o") return lin(w.o, s.heads * s.vdim, H_, 0, H_);
    if (rest == "mix.q.norm" && s.qk_norm != QKN_NONE) return vec(&w.q_norm, s.qk_norm == QKN_ALL ? nq : s.dim);
    if (rest == "mix.k.norm" && s.qk_norm != QKN_NONE) return vec(&w.k_norm, s.qk_norm == QKN_ALL ? nk : s.dim);
    if (rest == "mix.vmix") return vec(&w.v_mix, 1);
    if (rest == "mix.rel" && s.bias_reach > 0) {
        if (ndim != 2 || shape[1] != s.heads) return bad_shape();
        return w.rel ? twice() : load_bias_table(w, s, dtype, shape, host, nbytes);
    }
    if (s.mlp == MLP_MOE) {
        const int outs = s.experts + s.identity;
        if (rest == "mlp.correction") return vec(&w.correction, outs);
        if (rest == "mlp.router") {
            if (!is2(outs, H_)) return bad_shape();
            if (dtype != HM_BF16 || nbytes != n * 2) return fail(HM_ERR_UNSUPPORTED, "the router of this design must be stored as bf16");
            if (w.router) return twice();
            const int rc = stage(host, nbytes, reinterpret_cast<void**>(&w.router));
            if (rc) return rc;
            HM_CUDA(cudaStreamSynchronize(stream_));
            return HM_OK;
        }
        int rc = HM_OK;
        if (load_expert_tensor(w, s, name, rest, dtype, shape, ndim, host, nbytes, &rc)) return rc;
    }
    return fail(HM_ERR_INVALID, "unknown tensor name: " + name);
}

int Engine::finalize_gqa(const LayerW& w, const LayerSpec& s, const std::string& at) {
    if (w.in.loaded_parts != 3) return fail(HM_ERR_STATE, at + "mix.q / mix.k / mix.v");
    if (w.o.loaded_parts != 1) return fail(HM_ERR_STATE, at + "mix.o");
    if (s.qk_norm != QKN_NONE && (!w.q_norm || !w.k_norm)) return fail(HM_ERR_STATE, at + "mix.q.norm / mix.k.norm");
    if (s.bias_reach > 0 && !w.rel) return fail(HM_ERR_STATE, at + "mix.rel");
    if (s.v_first >= 0 && &w != &layers_[s.v_first] && !w.v_mix) return fail(HM_ERR_STATE, at + "mix.vmix");
    if (s.mlp != MLP_MOE) return HM_OK;
    if (!w.post_ln) return fail(HM_ERR_STATE, at + "norm2");
    if (!w.router || !w.correction) return fail(HM_ERR_STATE, at + "mlp.router / mlp.correction");
    for (int e = 0; e < s.experts; ++e)
        if ((size_t)e >= w.exp_seen.size() || w.exp_seen[e] != 7) return fail(HM_ERR_STATE, at + "mlp.e" + std::to_string(e));
    return HM_OK;
}

// ---- scratch ---------------------------------------------------------------------------------------

void Engine::free_gqa_scratch() {
    auto fr = [](auto*& p) {
        if (p) cudaFree(p);
        p = nullptr;
    };
    fr(sub_); fr(v_first_); fr(rt_ids_); fr(rt_weights_); fr(rt_identity_); fr(rt_dense_); fr(rt_mask_); fr(exp_act_); fr(exp_img_);
}

// A pass of a listed design has at most TC_ROWS rows.
int Engine::alloc_gqa_scratch() {
    if (!spec_.post_norm && !spec_.parallel) return HM_OK;
    size_t values = 1, top = 1, experts = 1, act = 1, img = 1;
    for (const LayerSpec& s : spec_.layers) {
        if (s.v_mix) values = std::max(values, (size_t)s.kv_heads * s.vdim);
        if (s.mlp != MLP_MOE) continue;
        top = std::max(top, (size_t)s.top);
        experts = std::max(experts, (size_t)s.experts);
        act = std::max(act, (size_t)s.top * expert_blocks(s.ff) * 64);
        img = std::max(img, (size_t)s.experts * tc_xpack_bytes(TC_ROWS, s.ff));
    }
    auto get = [&](auto** p, size_t count) -> cudaError_t {
        const cudaError_t e = cudaMalloc((void**)p, count * sizeof(**p));
        return e == cudaSuccess ? cudaMemset(*p, 0, count * sizeof(**p)) : e;
    };
    sub_parts_ = std::max(1, sm_count_ / ((H_ + SLAB - 1) / SLAB * 8));
    HM_CUDA(get(&sub_, (size_t)TC_ROWS * H_ * sub_parts_));
    HM_CUDA(get(&v_first_, TC_ROWS * values));
    HM_CUDA(get(&rt_ids_, TC_ROWS * top));
    HM_CUDA(get(&rt_weights_, TC_ROWS * top));
    HM_CUDA(get(&rt_identity_, TC_ROWS));
    HM_CUDA(get(&rt_dense_, TC_ROWS * experts));
    HM_CUDA(get(&rt_mask_, TC_ROWS * ((experts + 31) / 32)));
    HM_CUDA(get(&exp_act_, (use_tc_ ? MAX_M : TC_ROWS) * act));
    if (use_tc_) HM_CUDA(get(&exp_img_, img));
    return HM_OK;
}

GqaPool Engine::gqa_pool(int layer) const {
    const LayerSpec& s = spec_.layers[layer];
    return GqaPool{k_pool_[layer], v_pool_[layer], page_table_, max_pages_, s.kv_heads, s.dim, s.vdim, kv_bf16_ ? 1 : 0};
}

RouteOut Engine::route_out(bool dense) const { return RouteOut{rt_ids_, rt_weights_, rt_identity_, dense ? rt_dense_ : nullptr, rt_mask_}; }

// Experts that so many rows use, if their choices are spread evenly.
double Engine::experts_used(const LayerSpec& s, int rows) const { return s.experts * (1.0 - std::pow(1.0 - s.top / (double)(s.experts + s.identity), rows)); }

ExpertWeights Engine::expert_weights(int layer) const {
    const LayerSpec& s = spec_.layers[layer];
    return ExpertWeights{layers_[layer].exp_gu, layers_[layer].exp_down, s.experts, H_, s.ff, s.top, s.limit, s.act};
}

// Bytes of expert weights that the last profiled step read.
uint64_t Engine::expert_bytes(int layer, bool gate_up) const {
    if (!spec_.listed() || spec_.layers[layer].mlp != MLP_MOE || (int)experts_read_.size() <= layer) return 0;
    return (uint64_t)experts_read_[layer] * (gate_up ? 2 : 1) * spec_.layers[layer].ff * H_ * 2;
}

// Experts that the rows of the pass being enqueued have chosen (waits for the router).
int Engine::count_experts(int M, const LayerSpec& s) {
    std::vector<int32_t> ids((size_t)M * s.top);
    HM_CUDA(cudaMemcpyAsync(ids.data(), rt_ids_, ids.size() * 4, cudaMemcpyDeviceToHost, stream_));
    HM_CUDA(cudaStreamSynchronize(stream_));
    std::sort(ids.begin(), ids.end());
    int n = 0;
    for (size_t i = 0; i < ids.size(); ++i) n += ids[i] >= 0 && (i == 0 || ids[i] != ids[i - 1]);
    experts_seen_->push_back(n);
    return HM_OK;
}

// ---- shared pieces -----------------------------------------------------------------------------------

GqaRuns Engine::pass_runs(int M, int* longest) const {
    GqaRuns runs;
    *longest = 1;
    for (auto& r : pass_runs_) {
        runs.row[runs.n++] = (uint8_t)r.first;
        *longest = std::max(*longest, r.second);
    }
    runs.row[runs.n] = (uint8_t)M;
    return runs;
}

// The attention of layer l over the queries in q_, without what only some designs have and where the results go.
GqaAttnArgs Engine::gqa_attn_args(int l, int M, bool tall, const int32_t* row_pos, const int32_t* row_seq) const {
    GqaAttnArgs a{};
    a.pool = gqa_pool(l);
    a.q = q_;
    a.M = M;
    a.heads = spec_.layers[l].heads;
    a.row_pos = row_pos;
    a.row_seq = row_seq;
    a.runs = pass_runs(M, &a.longest_run);
    a.longest = pass_longest_;
    a.early = pass_runs_.empty() ? 1 : 0;  // the captured decode step
    a.max_cluster = use_clusters_ ? std::min(max_cluster_, 16) : 1;
    a.xp_mpad = tall ? tc_mpad(M) : 0;
    a.err_flag = err_flag_;
    return a;
}

int Engine::enqueue_experts(int l, int M, bool tall, const float* x, const float* resid, float* y, int* parts, int* launches) {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    auto want = [&](int cls) { return only_class_ < 0 || only_class_ == cls; };
    cudaError_t ce;
    TcArgs ta{};
    if (tall) {
        ta.ex.n = s.experts;
        ta.ex.blocks = expert_blocks(s.ff);
        ta.ex.weight = rt_dense_;
        ta.ex.mask = rt_mask_;
        ta.ex.limit = s.limit;
        ta.ex.act = s.act;
        ta.ex.img_bytes = tc_xpack_bytes(M, s.ff);
        ta.ex.used = std::max(1, (int)experts_used(s, M));
        ta.ex.parts = 1;
        ta.ex.part_stride = (size_t)TC_ROWS * H_;
        ta.M = M;
        ta.xp_mpad = tc_mpad(M);
        ta.err_flag = err_flag_;
    }
    if (want(PC_GATE_UP)) {
        if (tall) {
            TcArgs a = ta;
            a.W = w.exp_gu;
            a.K = H_;
            a.Kp = tc_padded_k(H_);
            a.N = s.experts * a.ex.blocks * SLAB;
            a.ksplit = tc_pick_split(H_, a.ex.used * a.ex.blocks * SLAB, sm_count_);
            a.xp = xpack_;
            a.epi = EPI_EXPERT;
            a.xp_out = exp_img_;
            ce = launch_gemm_tc(a, stream_, pdl_);
        } else {
            ce = launch_expert_gate_up(expert_weights(l), x, M, route_out(tall), exp_act_, stream_, pdl_);
        }
        if (ce != cudaSuccess) return cuda_fail(ce, "expert gate / up launch");
        ++*launches;
    }
    // the sum over the experts' activations is long: with few output blocks it is cut into parts, which the norm adds up
    const int down_k = ta.ex.used * expert_blocks(s.ff) * 64, down_split = tc_pick_split(down_k, H_, sm_count_);
    *parts = !tall ? 1 : std::max(1, std::min({sub_parts_, sm_count_ / ((H_ + SLAB - 1) / SLAB * down_split), down_k / 64 / (4 * down_split)}));
    if (want(PC_DOWN)) {
        if (tall) {
            TcArgs a = ta;
            a.W = w.exp_down;
            a.K = s.ff;
            a.Kp = tc_padded_k(s.ff);
            a.N = H_;
            a.ksplit = down_split;
            a.ex.parts = *parts;
            a.xp = exp_img_;
            a.epi = EPI_STORE;
            a.y = sub_;
            a.ldy = H_;
            ce = launch_gemm_tc(a, stream_, pdl_);
        } else {
            ce = launch_expert_down(expert_weights(l), exp_act_, M, route_out(tall), resid, y, stream_, pdl_);
        }
        if (ce != cudaSuccess) return cuda_fail(ce, "expert down launch");
        ++*launches;
    }
    return HM_OK;
}

// ---- one layer ---------------------------------------------------------------------------------------

int Engine::enqueue_gqa_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int next_lm_rows, int* launches) {
    const LayerW& w = layers_[l];
    const LayerSpec& s = spec_.layers[l];
    const float eps = (float)cfg_.rms_norm_eps;
    const bool tall = tall_rows(M);
    auto want = [&](int cls) { return only_class_ < 0 || only_class_ == cls; };
    auto prefetch = [&](const LinearW* n) {  // weights of the kernel two launches ahead (streaming passes)
        pf_ptr_ = nullptr;
        pf_bytes_ = 0;
        if (!use_prefetch_ || tall || only_class_ >= 0 || !n || !n->slabs) return;
        pf_ptr_ = n->slabs;
        pf_bytes_ = std::min(n->bytes(), (size_t)24 << 20);
    };
    cudaError_t ce;
    int rc = HM_OK;
    if (want(PC_QKV)) {
        if (tall) {
            if (l == 0) {  // later layers find the residual's image where the norm in front left it
                ce = launch_tc_pack_x(h_, H_, M, H_, nullptr, 0.f, xpack_, stream_, pdl_);
                if (ce != cudaSuccess) return cuda_fail(ce, "activation pack launch");
                ++*launches;
            }
            TcArgs a{};
            rc = enqueue_tc(w.in, M, xpack_, EPI_STORE, mix_raw_, qkv_ld(s), a, launches);
        } else {
            prefetch(&w.o);
            rc = enqueue_linear(w.in, M, h_, H_, PRO_PLAIN, nullptr, EPI_STORE, mix_raw_, qkv_ld(s), nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches);
        }
        if (rc) return rc;
    }
    if (want(PC_KV_WRITE)) {
        GqaPostArgs a{};
        a.pool = gqa_pool(l);
        a.raw = mix_raw_;
        a.ld = qkv_ld(s);
        a.M = M;
        a.heads = s.heads;
        a.qk_norm = s.qk_norm;
        a.q_norm = w.q_norm;
        a.k_norm = w.k_norm;
        a.eps = eps;
        a.q_scale = (float)(s.scale * 1.4426950408889634);
        a.temp_coef = s.temp_coef;
        a.temp_every = s.temp_every;
        a.v_first = s.v_first >= 0 ? v_first_ : nullptr;
        a.v_lambda = s.v_first >= 0 && s.v_first != l ? w.v_mix : nullptr;
        a.row_pos = row_pos;
        a.row_seq = row_seq;
        a.q_out = q_;
        ce = launch_gqa_post(a, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "query / key norm launch");
        ++*launches;
    }
    if (want(PC_ATTN)) {
        GqaAttnArgs a = gqa_attn_args(l, M, tall, row_pos, row_seq);
        a.bias = w.rel;
        a.reach = w.reach;
        a.out = attn_;
        if (tall) a.xp = xpack_attn_;
        ce = launch_gqa_attn(a, sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "attention launch");
        ++*launches;
    }
    if (want(PC_O)) {
        if (tall) {
            TcArgs a{};
            rc = enqueue_tc(w.o, M, xpack_attn_, EPI_STORE, sub_, H_, a, launches);
        } else {
            rc = enqueue_linear(w.o, M, attn_, s.heads * s.vdim, PRO_PLAIN, nullptr, EPI_STORE, sub_, H_, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches);
        }
        if (rc) return rc;
    }
    PostNormArgs pn{};
    pn.y = sub_;
    pn.x = h_;
    pn.M = M;
    pn.W = H_;
    pn.mult = spec_.residual_mult;
    pn.eps = eps;
    if (tall) {
        pn.xp = xpack_;
        pn.xp_mpad = tc_mpad(M);
    }
    const bool moe = s.mlp == MLP_MOE;
    if (want(moe ? PC_ROUTE : PC_NORM)) {
        PostNormArgs a = pn;
        a.w = w.in_ln;
        if (moe) {
            a.router = w.router;
            a.correction = w.correction;
            a.experts = s.experts;
            a.n_out = s.experts + s.identity;
            a.top = s.top;
            a.out = route_out(tall);
        }
        ce = launch_post_norm(a, sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "norm launch");
        ++*launches;
        if (experts_seen_ && moe) {
            rc = count_experts(M, s);
            if (rc) return rc;
        }
    }
    if (!moe) return HM_OK;
    int parts = 1;
    rc = enqueue_experts(l, M, tall, h_, nullptr, sub_, &parts, launches);
    if (rc) return rc;
    if (want(PC_NORM)) {
        PostNormArgs a = pn;
        a.w = w.post_ln;
        a.parts = parts;
        a.part_stride = (size_t)TC_ROWS * H_;
        a.identity = s.identity > 0 ? rt_identity_ : nullptr;
        ce = launch_post_norm(a, sm_count_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "norm launch");
        ++*launches;
    }
    return HM_OK;
}

}  // namespace hm
