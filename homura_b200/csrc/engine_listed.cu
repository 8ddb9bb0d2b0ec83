// Engine parts for designs that list their layers (ModelSpec::layers): weight loading, scratch and cache of latent attention,
// and the launches of one layer.  The projections, the captured decode step, the sampler and the cache bookkeeping are the
// ones every design uses (engine.cu, engine_step.cu).
//
// A layer of latent attention with an MLP is, per pass,
//   in      [queries | output gate | latents]  <- grouped norm + token shift of the residual
//   write   normalised latents -> page slots                         (layers with latents of their own)
//   kup     per head: query into latent space (the key up-projection, transposed)
//   attn    softmax over latents, result in latent space             (latent_attn.cu)
//   vup     per head: result -> values, times sigmoid(gate)
//   o       output projection, layer scale, residual
//   up      grouped norm, projection, squared ReLU;   down  projection, layer scale, residual
// Passes of a few rows run the streaming kernel with the norm in its prologue; larger passes run the tensor-core GEMM on
// packed activations, which the producers write themselves wherever the sizes allow.
#include <algorithm>

#include "engine.h"
#include "engine_parallel.h"
#include "engine_util.h"
#include "gemm_tc.h"

namespace hm {

namespace {
int pad128(int n) { return (n + 127) / 128 * 128; }
int in_gate(const LayerSpec& s) { return pad128(s.heads * s.dim); }                     // first column of the gate in the input projection
int in_latent(const LayerSpec& s) { return in_gate(s) + pad128(s.heads * s.vdim); }     // first column of the latents
int in_cols(const LayerSpec& s) { return in_latent(s) + (s.kv_from < 0 ? s.kv_rank : 0); }
int in_ld(const LayerSpec& s) { return (in_cols(s) + 3) / 4 * 4; }
}  // namespace

// ---- weights -----------------------------------------------------------------------------------

// One [group_n, K] matrix per group (or, src_is_kn, [K, group_n]: applied transposed), stacked in `host`.
int Engine::load_grouped(LinearW& L, int groups, int K, int group_n, bool src_is_kn, int dtype, const void* host, size_t nbytes) {
    if (dtype != HM_BF16) return fail(HM_ERR_UNSUPPORTED, "projection weights of this design must be stored as bf16");
    const size_t elems = (size_t)groups * K * group_n;
    if (nbytes != elems * 2) return fail(HM_ERR_INVALID, "tensor byte size does not match its shape");
    L.K = K;
    L.groups = groups;
    L.group_n = group_n;
    L.group_slabs = (group_n + SLAB - 1) / SLAB;
    L.N = groups * group_n;
    L.kind = HM_BF16;
    cfg_.weight_dtype = HM_BF16;
    void* tmp = nullptr;
    int rc = stage(host, nbytes, &tmp);
    if (rc) return rc;
    const size_t slab_elems = (size_t)groups * L.group_slabs * K * SLAB;
    cudaError_t ce = cudaMalloc(&L.slabs, slab_elems * 2);
    if (ce == cudaSuccess) ce = cudaMemsetAsync(L.slabs, 0, slab_elems * 2, stream_);
    if (use_tc_) {
        const size_t bytes = tc_packed_elems(K, L.columns()) * 2;
        if (ce == cudaSuccess) ce = cudaMalloc(&L.tc, bytes);
        if (ce == cudaSuccess) ce = cudaMemsetAsync(L.tc, 0, bytes, stream_);
    }
    for (int g = 0; g < groups && ce == cudaSuccess; ++g) {
        const uint16_t* src = (const uint16_t*)tmp + (size_t)g * K * group_n;
        const int n_off = g * L.group_slabs * SLAB;
        ce = src_is_kn ? launch_pack_slabs_from_kn(src, K, group_n, L.slabs + (size_t)n_off * K, stream_) : launch_pack_slabs_from_nk(src, group_n, K, L.slabs, n_off, -1, stream_);
        if (use_tc_ && ce == cudaSuccess) ce = launch_pack_tc(src, group_n, K, src_is_kn, L.tc, n_off, -1, stream_);
    }
    if (ce == cudaSuccess) ce = cudaStreamSynchronize(stream_);
    cudaFree(tmp);
    if (ce != cudaSuccess) return cuda_fail(ce, "load_grouped");
    L.loaded_parts++;
    return HM_OK;
}

int Engine::load_listed_tensor(const std::string& name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes) {
    size_t n = 1;
    for (int i = 0; i < ndim; ++i) n *= (size_t)shape[i];
    auto is2 = [&](int64_t a, int64_t b) { return ndim == 2 && shape[0] == a && shape[1] == b; };
    auto bad_shape = [&]() { return fail(HM_ERR_INVALID, "unexpected shape for tensor " + name); };
    auto vec = [&](float** dst, int len) {
        if (ndim != 1 || shape[0] != len) return bad_shape();
        if (*dst) return fail(HM_ERR_STATE, "tensor loaded twice: " + name);
        return load_vec_f32(dst, len, 0, dtype, host, n, nbytes);
    };
    auto lin = [&](LinearW& L, int K, int total, int off, int part) { return is2(part, K) ? load_linear(L, K, total, off, part, -1, dtype, host, nbytes) : bad_shape(); };
    auto grouped = [&](LinearW& L, int groups, int K, int group_n, bool kn, int64_t rows, int64_t cols) {
        if (!is2(rows, cols)) return bad_shape();
        if (L.loaded_parts) return fail(HM_ERR_STATE, "tensor loaded twice: " + name);
        return load_grouped(L, groups, K, group_n, kn, dtype, host, nbytes);
    };
    if (name == "embed") {
        if (!is2(V_, H_)) return bad_shape();
        if (embed_) return fail(HM_ERR_STATE, "embedding loaded twice");
        if (dtype != HM_BF16 || nbytes != n * 2) return fail(HM_ERR_UNSUPPORTED, "the embedding of this design must be stored as bf16");
        const int rc = stage(host, nbytes, &embed_);
        if (rc) return rc;
        HM_CUDA(cudaStreamSynchronize(stream_));
        embed_dtype_ = HM_BF16;
        return cfg_.tie_word_embeddings ? lin(lm_head_, H_, V_, 0, V_) : HM_OK;
    }
    if (name == "final.norm") {
        const int rc = vec(&final_norm_, H_);
        if (rc == HM_OK && spec_.norm_offset) HM_CUDA(launch_add_constant(final_norm_, H_, 1.f, stream_));
        return rc;
    }
    if (name == "bigram" && spec_.bigram_buckets > 0) return load_bigram(dtype, shape, ndim, host, nbytes);
    if (name == "head" && cfg_.tie_word_embeddings) return fail(HM_ERR_INVALID, "unknown tensor name: " + name);
    if (name == "head") return lin(lm_head_, H_, V_, 0, V_);
    const size_t dot = name.find('.');
    if (name.size() < 3 || name[0] != 'l' || dot == std::string::npos || name.find_first_not_of("0123456789", 1) != dot) return fail(HM_ERR_INVALID, "unknown tensor name: " + name);
    const long li = std::atol(name.c_str() + 1);
    if (li < 0 || li >= L_) return fail(HM_ERR_INVALID, "layer index out of range in " + name);
    const std::string rest = name.substr(dot + 1);
    LayerW& w = layers_[li];
    const LayerSpec& s = spec_.layers[li];
    if (rest == "norm1") {
        const int rc = vec(&w.in_ln, H_);
        if (rc == HM_OK && spec_.norm_offset) HM_CUDA(launch_add_constant(w.in_ln, H_, 1.f, stream_));
        return rc;
    }
    if (spec_.sandwich) return load_sandwich_tensor((int)li, name, rest, dtype, shape, ndim, host, nbytes);
    if (spec_.parallel) return load_parallel_tensor((int)li, name, rest, dtype, shape, ndim, host, nbytes);
    if (rest == "norm2") return vec(&w.post_ln, H_);
    if (s.mixer == MIX_GQA) return load_gqa_tensor(w, s, name, rest, dtype, shape, ndim, host, nbytes);
    if (rest == "shift") return vec(&w.shift, H_);
    if (rest == "ls1") return vec(&w.ls1, H_);
    if (rest == "ls2") return vec(&w.ls2, H_);
    if (rest == "mix.q") return lin(w.in, H_, in_cols(s), 0, s.heads * s.dim);
    if (rest == "mix.g") return lin(w.in, H_, in_cols(s), in_gate(s), s.heads * s.vdim);
    if (rest == "mix.dkv" && s.kv_from < 0) return lin(w.in, H_, in_cols(s), in_latent(s), s.kv_rank);
    if (rest == "mix.dkv.norm" && s.kv_from < 0) return vec(&w.latent_norm, s.kv_rank);
    // keys are W_uk c, so a query meets the latents as W_uk^T q
    if (rest == "mix.uk") return grouped(w.kup, s.heads, s.dim, s.kv_rank, true, (int64_t)s.heads * s.dim, s.kv_rank);
    if (rest == "mix.uv") return grouped(w.vup, s.heads, s.kv_rank, s.vdim, false, (int64_t)s.heads * s.vdim, s.kv_rank);
    if (rest == "mix.o") return lin(w.o, s.heads * s.vdim, H_, 0, H_);
    if (rest == "mlp.up" && s.mlp == MLP_SQRELU) return lin(w.gu, H_, s.ff, 0, s.ff);
    if (rest == "mlp.down" && s.mlp == MLP_SQRELU) return lin(w.down, s.ff, H_, 0, H_);
    return fail(HM_ERR_INVALID, "unknown tensor name: " + name);
}

int Engine::finalize_listed() {
    if (spec_.sandwich) return finalize_sandwich();
    if (spec_.parallel) return finalize_parallel();
    for (int i = 0; i < L_; ++i) {
        const LayerW& l = layers_[i];
        const LayerSpec& s = spec_.layers[i];
        const std::string p = "missing weight in layer " + std::to_string(i) + ": ";
        if (!l.in_ln) return fail(HM_ERR_STATE, p + "norm1");
        if (s.mixer == MIX_GQA) {
            const int rc = finalize_gqa(l, s, p);
            if (rc) return rc;
            continue;
        }
        if (spec_.token_shift && !l.shift) return fail(HM_ERR_STATE, p + "shift");
        if (spec_.layer_scale && !l.ls1) return fail(HM_ERR_STATE, p + "ls1");
        if (l.in.loaded_parts != (s.kv_from < 0 ? 3 : 2)) return fail(HM_ERR_STATE, p + "mix.q / mix.g / mix.dkv");
        if (s.kv_from < 0 && !l.latent_norm) return fail(HM_ERR_STATE, p + "mix.dkv.norm");
        if (!l.kup.loaded_parts || !l.vup.loaded_parts) return fail(HM_ERR_STATE, p + "mix.uk / mix.uv");
        if (l.o.loaded_parts != 1) return fail(HM_ERR_STATE, p + "mix.o");
        if (s.mlp == MLP_NONE) continue;
        if (!l.post_ln || (spec_.layer_scale && !l.ls2)) return fail(HM_ERR_STATE, p + "norm2 / ls2");
        if (l.gu.loaded_parts != 1 || l.down.loaded_parts != 1) return fail(HM_ERR_STATE, p + "mlp.up / mlp.down");
    }
    return HM_OK;
}

// ---- scratch and cache -----------------------------------------------------------------------------

void Engine::free_listed() {
    auto fr = [](auto*& p) {
        if (p) cudaFree(p);
        p = nullptr;
    };
    free_gqa_scratch();
    free_parallel_scratch();
    fr(mix_raw_); fr(qlat_); fr(ctx_); fr(xpack_q_); fr(xpack_ctx_); fr(lat_acc_); fr(lat_ml_);
}

int Engine::alloc_listed_scratch(int cap) {
    free_listed();
    size_t raw = 1, lat = 1, q_img = 1, ctx_img = 1, acc = 1, ml = 1;
    int kmax = H_;
    for (const LayerSpec& s : spec_.layers) {
        kmax = std::max(kmax, std::max(s.heads * s.vdim, s.ff));
        if (spec_.parallel) raw = std::max(raw, (size_t)parallel_columns(s).ld);
        if (spec_.sandwich) raw = std::max(raw, (size_t)sandwich_columns(s).ld);
        if (s.mixer != MIX_LATENT) {
            raw = std::max(raw, (size_t)(s.heads * s.dim + s.kv_heads * (s.dim + s.vdim) + 3) / 4 * 4);
            continue;
        }
        raw = std::max(raw, (size_t)in_ld(s));
        const int rank = s.latent_rank();
        lat = std::max(lat, (size_t)s.heads * rank);
        q_img = std::max(q_img, s.heads * tc_xpack_bytes(TC_ROWS, s.rot_dim ? s.q_stride() : s.dim));
        ctx_img = std::max(ctx_img, s.heads * tc_xpack_bytes(TC_ROWS, rank));
        kmax = std::max(kmax, std::max(s.dim, rank));
        // splits times rows never exceed the SMs times the rows that share a CTA (latent_pick_nsplit)
        for (int bf16 = 0; bf16 < 2; ++bf16) {
            const size_t rows = 2 * (size_t)sm_count_ * latent_rows_per_tile(TC_ROWS, 1 << 30, s.heads, rank, bf16);
            acc = std::max(acc, rows * s.heads * rank);
            ml = std::max(ml, rows * s.heads * 2);
        }
    }
    auto get = [&](auto** p, size_t count) -> cudaError_t {
        if (*p) cudaFree(*p);
        *p = nullptr;
        cudaError_t e = cudaMalloc((void**)p, count * sizeof(**p));
        if (e == cudaSuccess) e = cudaMemset(*p, 0, count * sizeof(**p));
        return e;
    };
    HM_CUDA(get(&mix_raw_, raw * cap));
    HM_CUDA(get(&qlat_, lat * cap));
    HM_CUDA(get(&ctx_, lat * cap));
    HM_CUDA(get(&lat_acc_, acc));
    HM_CUDA(get(&lat_ml_, ml));
    lat_acc_floats_ = acc;
    lat_ml_floats_ = ml;
    if (use_tc_) {
        xpack_bytes_ = tc_xpack_bytes(TC_ROWS, kmax);
        HM_CUDA(get(&xpack_, xpack_bytes_));
        HM_CUDA(get(&xpack_attn_, tc_xpack_bytes(TC_ROWS, qdim_)));
        HM_CUDA(get(&xpack_act_, tc_xpack_bytes(TC_ROWS, I_)));
        HM_CUDA(get(&xpack_q_, q_img));
        HM_CUDA(get(&xpack_ctx_, ctx_img));
    }
    int rc = alloc_gqa_scratch();
    if (rc == HM_OK) rc = alloc_parallel_scratch();
    return rc ? rc : alloc_sandwich_scratch();
}

void Engine::free_listed_cache() {
    for (void* p : lat_pool_)
        if (p) cudaFree(p);
    lat_pool_.clear();
    if (shift_state_) cudaFree(shift_state_);
    if (shift_saved_) cudaFree(shift_saved_);
    shift_state_ = shift_saved_ = nullptr;
    if (state_) cudaFree(state_);
    if (state_saved_) cudaFree(state_saved_);
    state_ = state_saved_ = nullptr;
}

int Engine::alloc_listed_cache(int batch, size_t n_pages) {
    lat_pool_.assign(L_, nullptr);
    for (int l = 0; l < L_; ++l) {
        const LayerSpec& s = spec_.layers[l];
        if (s.paged_kv()) {
            const size_t esz = kv_bf16_ ? 2 : 4, kb = n_pages * gqa_page_elems(s.kv_heads, s.dim) * esz, vb = n_pages * gqa_page_elems(s.kv_heads, s.vdim) * esz;
            HM_CUDA(cudaMalloc(&k_pool_[l], kb));
            HM_CUDA(cudaMalloc(&v_pool_[l], vb));
            HM_CUDA(cudaMemset(k_pool_[l], 0, kb));
            HM_CUDA(cudaMemset(v_pool_[l], 0, vb));
            continue;
        }
        if (s.mixer != MIX_LATENT || s.kv_from >= 0) continue;
        const size_t bytes = n_pages * latent_page_elems(s.latent_rank(), kv_bf16_) * (kv_bf16_ ? 2 : 4);
        HM_CUDA(cudaMalloc(&lat_pool_[l], bytes));
        HM_CUDA(cudaMemset(lat_pool_[l], 0, bytes));
    }
    state_floats_ = 0;
    for (int l = 0; l < L_; ++l) {
        const LayerSpec& s = spec_.layers[l];
        LayerW& w = layers_[l];
        w.conv_at = state_floats_;
        if (s.conv > 1) state_floats_ += ((size_t)conv_slots(s.conv) * (s.heads * s.dim + s.kv_heads * (s.dim + (s.tied_values ? 0 : s.vdim))) + 3) / 4 * 4;
        w.lin_conv_at = state_floats_;
        if (s.lin_conv > 1) state_floats_ += ((size_t)conv_slots(s.lin_conv) * s.lin_channels() + 3) / 4 * 4;
        w.gla_at = state_floats_;
        if (s.linear()) state_floats_ += s.lin_heads * gla_state_floats(s.lin_dim, s.lin_vdim);
    }
    if (state_floats_) {
        HM_CUDA(cudaMalloc(&state_, batch * state_floats_ * 4));
        HM_CUDA(cudaMemset(state_, 0, batch * state_floats_ * 4));
        HM_CUDA(cudaMalloc(&state_saved_, state_floats_ * 4));
    }
    if (spec_.token_shift) {
        const size_t row = (size_t)SHIFT_RING * H_ * 4;
        HM_CUDA(cudaMalloc(&shift_state_, (size_t)L_ * batch * row));
        HM_CUDA(cudaMemset(shift_state_, 0, (size_t)L_ * batch * row));
        HM_CUDA(cudaMalloc(&shift_saved_, (size_t)L_ * row));
    }
    return HM_OK;
}

LatentPool Engine::latent_pool(int layer) const {
    const LayerSpec& s = spec_.layers[layer];
    return LatentPool{lat_pool_[s.kv_from >= 0 ? s.kv_from : layer], page_table_, max_pages_, s.latent_rank(), kv_bf16_ ? 1 : 0};
}

int Engine::latent_view(int seq, int layer, float* out) {
    if (!set_device()) return fail(HM_ERR_CUDA, "cudaSetDevice failed");
    if (batch_ == 0) return fail(HM_ERR_STATE, "latent_view before kv_alloc");
    if (seq < 0 || seq >= batch_ || layer < 0 || layer >= L_ || !out) return fail(HM_ERR_INVALID, "latent_view: bad arguments");
    if (!spec_.listed() || spec_.layers[layer].mixer != MIX_LATENT) return fail(HM_ERR_UNSUPPORTED, "latent_view: this design caches keys and values (hm_kv_view)");
    const int len = len_[seq];
    if (len == 0) return HM_OK;
    const size_t bytes = (size_t)len * spec_.layers[layer].latent_rank() * 4;
    float* d = nullptr;
    HM_CUDA(cudaMalloc(&d, bytes));
    cudaError_t ce = launch_latent_read(latent_pool(layer), seq, len, d, stream_);
    if (ce == cudaSuccess) ce = cudaMemcpyAsync(out, d, bytes, cudaMemcpyDeviceToHost, stream_);
    if (ce == cudaSuccess) ce = cudaStreamSynchronize(stream_);
    cudaFree(d);
    if (ce != cudaSuccess) return cuda_fail(ce, "latent_view");
    return HM_OK;
}

int Engine::save_state(int seq) {
    if (state_) HM_CUDA(cudaMemcpyAsync(state_saved_, state_ + seq * state_floats_, state_floats_ * 4, cudaMemcpyDeviceToDevice, stream_));
    if (!shift_state_) return HM_OK;
    const size_t row = (size_t)SHIFT_RING * H_ * 4;
    HM_CUDA(cudaMemcpy2DAsync(shift_saved_, row, reinterpret_cast<char*>(shift_state_) + seq * row, batch_ * row, row, L_, cudaMemcpyDeviceToDevice, stream_));
    return HM_OK;
}

// Back to `len` tokens plus the tokens of `fed`.  A cache addressed by position only forgets its length; state that is not
// is restored from save_state() (taken at `len` tokens) and the tokens of `fed` are run again.  One-sequence engines only.
int Engine::rewind(int seq, int len, const std::vector<uint32_t>& fed) {
    const int target = len + (int)fed.size();
    if (len_[seq] == target) return HM_OK;
    if (!shift_state_ && !state_) {
        len_[seq] = target;
        HM_CUDA(cudaMemcpy(pos_dev_ + seq, &len_[seq], 4, cudaMemcpyHostToDevice));
        return HM_OK;
    }
    const size_t row = (size_t)SHIFT_RING * H_ * 4;
    if (state_) HM_CUDA(cudaMemcpyAsync(state_ + seq * state_floats_, state_saved_, state_floats_ * 4, cudaMemcpyDeviceToDevice, stream_));
    if (shift_state_) HM_CUDA(cudaMemcpy2DAsync(reinterpret_cast<char*>(shift_state_) + seq * row, batch_ * row, shift_saved_, row, row, L_, cudaMemcpyDeviceToDevice, stream_));
    HM_CUDA(cudaStreamSynchronize(stream_));
    HM_CUDA(cudaMemcpy(pos_dev_ + seq, &len, 4, cudaMemcpyHostToDevice));
    for (uint32_t t : fed) {
        HM_CUDA(cudaMemcpy(tokens_dev_ + seq, &t, 4, cudaMemcpyHostToDevice));
        HM_CUDA(launch_hist_set(tokens_dev_, pos_dev_, hist_dev_, max_seq_ + 1, batch_, stream_));
        const int rc = launch_step();
        if (rc) return rc;
        HM_CUDA(cudaStreamSynchronize(stream_));
    }
    len_[seq] = target;
    return HM_OK;
}

// ---- one layer ------------------------------------------------------------------------------------------

// Tensor-core projection of up to 64 packed rows; `a` carries what the epilogue needs beyond the common arguments.
int Engine::enqueue_tc(const LinearW& L, int M, const unsigned char* xp, int epi, float* y, int ldy, TcArgs& a, int* launches) {
    if (!L.tc) return fail(HM_ERR_STATE, "tensor-core weight copy missing");
    a.W = L.tc;
    a.K = L.K;
    a.Kp = tc_padded_k(L.K);
    a.N = L.N;
    a.M = M;
    a.ksplit = tc_pick_split(L.K, L.columns(), sm_count_);
    if (L.groups)  // short contractions over few blocks: half as many k-blocks per CTA as the wide projections keep
        while (a.ksplit < 4 && a.Kp / 64 / (a.ksplit * 2) >= 2 && L.columns() / SLAB * a.ksplit * 2 <= sm_count_) a.ksplit *= 2;
    a.xp = xp;
    a.xp_mpad = tc_mpad(M);
    a.epi = epi;
    a.y = y;
    a.ldy = ldy;
    if (L.groups) {
        a.group_blocks = L.group_slabs;
        a.group_n = L.group_n;
        a.group_xp = tc_xpack_bytes(M, L.K);
    }
    a.err_flag = err_flag_;
    const cudaError_t ce = launch_gemm_tc(a, stream_, pdl_);
    if (ce != cudaSuccess) return cuda_fail(ce, "tensor-core projection launch");
    ++*launches;
    return HM_OK;
}

// Attention of layer l over the queries in latent space (qlat_) into ctx_ or, many rows, its images; pass_nsplit_ splits are left to the next projection.
int Engine::enqueue_latent_attn(int l, int M, bool tall, const int32_t* row_pos, const int32_t* row_seq, int* launches) {
    const LayerSpec& s = spec_.layers[l];
    const int rank = s.latent_rank(), lat = s.heads * rank;
    LatentAttnArgs a{};
    a.pool = latent_pool(l);
    a.q = qlat_;
    a.ldq = lat;
    a.M = M;
    a.heads = s.heads;
    a.row_pos = row_pos;
    a.row_seq = row_seq;
    a.scale = s.scale;
    a.window = s.window;
    const size_t per = (size_t)M * s.heads;
    const int most = (int)std::min<size_t>(std::min(lat_acc_floats_ / (per * rank), lat_ml_floats_ / (per * 2)), 256);
    // tiles: every run is cut at the multiples of the rows that share a CTA
    int longest_run = 1, tiles = 0;
    for (auto& r : pass_runs_) longest_run = std::max(longest_run, r.second);
    const int longest = s.window > 0 ? (int)std::min((long)pass_longest_, (long)s.window + longest_run + 62) : pass_longest_;  // tokens that a tile's pages range over
    a.rows_per_tile = latent_rows_per_tile(longest_run, longest, s.heads, rank, kv_bf16_);
    for (auto& r : pass_runs_) tiles += (r.first + r.second - 1) / a.rows_per_tile - r.first / a.rows_per_tile + 1;
    if (a.rows_per_tile == 1) tiles = M;
    a.tiles = tiles;
    a.unmerged = !tall && rank % 4 == 0 ? 1 : 0;
    a.early = pass_runs_.empty() ? 1 : 0;  // the captured decode step
    a.nsplit = latent_pick_nsplit(tiles, a.rows_per_tile, s.heads, rank, kv_bf16_, longest, sm_count_, most, a.unmerged != 0);
    pass_nsplit_ = a.unmerged ? a.nsplit : 1;
    a.part_acc = lat_acc_;
    a.part_ml = lat_ml_;
    a.out = ctx_;
    a.ldo = lat;
    if (tall) {
        a.xp = xpack_ctx_;
        a.xp_mpad = tc_mpad(M);
        a.xp_bytes = tc_xpack_bytes(M, rank);
    }
    a.err_flag = err_flag_;
    const cudaError_t ce = launch_latent_attn(a, stream_, pdl_, launches);
    if (ce != cudaSuccess) return cuda_fail(ce, "latent attention launch");
    return HM_OK;
}

int Engine::enqueue_listed_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int next_lm_rows, int* launches) {
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
    RowNorm gn{};
    gn.groups = spec_.norm_groups;
    if (spec_.token_shift) {
        gn.shift = w.shift;
        gn.state = shift_state_ + (size_t)l * batch_ * SHIFT_RING * H_;
        gn.row_pos = row_pos;
        gn.row_seq = row_seq;
    }
    RowNorm gn2{};
    gn2.groups = spec_.norm_groups;
    const int ld = in_ld(s), lat = s.heads * s.kv_rank, vals = s.heads * s.vdim;
    const float *gate = mix_raw_ + in_gate(s), *raw_c = mix_raw_ + in_latent(s);

    // queries, gate, latents
    if (want(PC_QKV)) {
        if (tall) {
            ce = launch_tc_pack_gnorm(h_, H_, M, H_, w.in_ln, eps, gn, xpack_, stream_, pdl_);
            if (ce != cudaSuccess) return cuda_fail(ce, "norm and pack launch");
            ++*launches;
            TcArgs a{};
            const bool direct = s.dim % 8 == 0;  // queries leave as the images the next projection reads
            if (direct) {
                a.split_xp = xpack_q_;
                a.split_n = s.heads * s.dim;
                a.split_k = s.dim;
                a.split_bytes = tc_xpack_bytes(M, s.dim);
            }
            rc = enqueue_tc(w.in, M, xpack_, EPI_STORE, mix_raw_, ld, a, launches);
            if (rc) return rc;
            if (!direct) {
                ce = launch_tc_pack_x(mix_raw_, ld, M, s.dim, nullptr, 0.f, xpack_q_, stream_, pdl_, nullptr, s.heads, s.dim, tc_xpack_bytes(M, s.dim));
                if (ce != cudaSuccess) return cuda_fail(ce, "query pack launch");
                ++*launches;
            }
        } else {
            LinOpt o;
            o.gn = gn;
            prefetch(&w.vup);
            rc = enqueue_linear(w.in, M, h_, H_, PRO_GNORM, w.in_ln, EPI_STORE, mix_raw_, ld, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
            if (rc) return rc;
        }
    }
    if (want(PC_LATENT) && s.kv_from < 0) {
        ce = launch_latent_write(latent_pool(l), raw_c, ld, M, w.latent_norm, eps, row_pos, row_seq, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "latent write launch");
        ++*launches;
    }
    if (want(PC_KUP)) {
        if (tall) {
            TcArgs a{};
            rc = enqueue_tc(w.kup, M, xpack_q_, EPI_STORE, qlat_, lat, a, launches);
        } else {
            LinOpt o;
            o.group_x = s.dim;
            prefetch(&w.o);
            rc = enqueue_linear(w.kup, M, mix_raw_, ld, PRO_PLAIN, nullptr, EPI_STORE, qlat_, lat, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
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
            a.gate = gate;
            a.ld_gate = ld;
            a.xp_out = xpack_attn_;
            rc = enqueue_tc(w.vup, M, xpack_ctx_, EPI_GATE, attn_, vals, a, launches);
        } else {
            LinOpt o;
            o.group_x = s.kv_rank;
            o.gate = gate;
            o.ld_gate = ld;
            const bool merge = pass_nsplit_ > 1;
            if (merge) o.split = SplitRows{lat_acc_, lat_ml_, pass_nsplit_, s.heads};
            prefetch(s.mlp == MLP_NONE ? nullptr : &w.gu);
            rc = enqueue_linear(w.vup, M, ctx_, lat, merge ? PRO_MERGE : PRO_PLAIN, nullptr, EPI_GATE, attn_, vals, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    const LinearW* next_in = l + 1 < L_ ? &layers_[l + 1].in : (next_lm_rows > 0 ? &lm_head_ : nullptr);
    if (want(PC_O)) {
        if (tall) {
            TcArgs a{};
            a.out_scale = w.ls1;
            a.resid = h_;
            rc = enqueue_tc(w.o, M, xpack_attn_, EPI_STORE, h_, H_, a, launches);
        } else {
            LinOpt o;
            o.out_scale = w.ls1;
            prefetch(s.mlp == MLP_NONE ? nullptr : &w.down);
            rc = enqueue_linear(w.o, M, attn_, vals, PRO_PLAIN, nullptr, EPI_STORE, h_, H_, nullptr, h_, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    if (s.mlp == MLP_NONE) return HM_OK;
    if (want(PC_GATE_UP)) {
        if (tall) {
            ce = launch_tc_pack_gnorm(h_, H_, M, H_, w.post_ln, eps, gn2, xpack_, stream_, pdl_);
            if (ce != cudaSuccess) return cuda_fail(ce, "norm and pack launch");
            ++*launches;
            TcArgs a{};
            a.xp_out = xpack_act_;
            rc = enqueue_tc(w.gu, M, xpack_, EPI_SQRELU, act_, s.ff, a, launches);
        } else {
            LinOpt o;
            o.gn = gn2;
            prefetch(next_in);
            rc = enqueue_linear(w.gu, M, h_, H_, PRO_GNORM, w.post_ln, EPI_SQRELU, act_, s.ff, nullptr, nullptr, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    if (want(PC_DOWN)) {
        if (tall) {
            TcArgs a{};
            a.out_scale = w.ls2;
            a.resid = h_;
            rc = enqueue_tc(w.down, M, xpack_act_, EPI_STORE, h_, H_, a, launches);
        } else {
            LinOpt o;
            o.out_scale = w.ls2;
            prefetch(l + 1 < L_ ? &layers_[l + 1].kup : nullptr);
            rc = enqueue_linear(w.down, M, act_, s.ff, PRO_PLAIN, nullptr, EPI_STORE, h_, H_, nullptr, h_, l, row_pos, row_seq, nullptr, nullptr, launches, nullptr, &o);
        }
        if (rc) return rc;
    }
    return HM_OK;
}

// Final norm and LM head over `rows` rows of x into dst [rows][V] (argmax as in the uniform designs).
int Engine::enqueue_listed_logits(const float* x, int rows, float* dst, const ArgmaxFold& fold, int* launches) {
    RowNorm gn{};
    gn.groups = spec_.norm_groups;
    const float eps = (float)cfg_.rms_norm_eps;
    if (tall_rows(rows)) {
        const cudaError_t ce = launch_tc_pack_gnorm(x, H_, rows, H_, final_norm_, eps, gn, xpack_, stream_, pdl_);
        if (ce != cudaSuccess) return cuda_fail(ce, "norm and pack launch");
        ++*launches;
        TcArgs a{};
        a.amax_val = amax_val_;
        a.amax_idx = amax_idx_;
        a.softcap = spec_.softcap;
        return enqueue_tc(lm_head_, rows, xpack_, EPI_LOGITS, dst, V_, a, launches);
    }
    LinOpt o;
    o.gn = gn;
    o.softcap = spec_.softcap;
    return enqueue_linear(lm_head_, rows, x, H_, PRO_GNORM, final_norm_, EPI_LOGITS, dst, V_, nullptr, nullptr, -1, nullptr, nullptr, amax_val_, amax_idx_, launches, &fold, &o);
}

}  // namespace hm
