// Pages shared by the sequences of an engine, and the step over portions of several sequences (every design).
#include <algorithm>
#include <cstring>
#include <vector>

#include "engine.h"
#include "engine_util.h"
#include "gemm_tc.h"

namespace hm {

// ---- pages ------------------------------------------------------------------------------------------

// Gives every listed sequence the pages for the tokens it will hold.  All or nothing: HM_ERR_KV_FULL when the pool is short.
int Engine::ensure_pages(const std::vector<std::pair<int, long>>& need) {
    if (!pooled_) return HM_OK;
    size_t missing = 0;
    for (auto& n : need) {
        const size_t pages = (size_t)(n.second + page_tokens_ - 1) / page_tokens_, have = seq_pages_[n.first].size();
        if (pages > (size_t)max_pages_) return fail(HM_ERR_KV_FULL, "KV cache full (sequence longer than max_seq_len)");
        if (pages > have) missing += pages - have;
    }
    if (missing > free_pages_.size())
        return fail(HM_ERR_KV_FULL, "KV cache full (" + std::to_string(missing) + " more pages wanted, " + std::to_string(free_pages_.size()) + " free in the pool)");
    for (auto& n : need) {
        std::vector<int32_t>& own = seq_pages_[n.first];
        const size_t pages = (size_t)(n.second + page_tokens_ - 1) / page_tokens_, first = own.size();
        if (pages <= first) continue;
        for (size_t i = first; i < pages; ++i) {
            own.push_back(free_pages_.back());
            free_pages_.pop_back();
        }
        HM_CUDA(cudaMemcpyAsync(page_table_ + (size_t)n.first * max_pages_ + first, own.data() + first, (pages - first) * 4, cudaMemcpyHostToDevice, stream_));
    }
    return HM_OK;
}

int Engine::ensure_pages_all(int more) {
    if (!pooled_) return HM_OK;
    std::vector<std::pair<int, long>> need;
    for (int b = 0; b < batch_; ++b) need.push_back({b, (long)len_[b] + more});
    return ensure_pages(need);
}

void Engine::release_pages(int seq) {
    if (!pooled_) return;
    std::vector<int32_t>& own = seq_pages_[seq];
    while (!own.empty()) {
        free_pages_.push_back(own.back());
        own.pop_back();
    }
}

int Engine::kv_free_tokens(long* out) {
    if (!out) return fail(HM_ERR_INVALID, "kv_free_tokens: null output");
    if (batch_ == 0 || !pooled_) return fail(HM_ERR_STATE, "kv_free_tokens: the cache has no shared pool");
    *out = (long)free_pages_.size() * page_tokens_;
    return HM_OK;
}

// ---- step ---------------------------------------------------------------------------------------------

int Engine::tap(int layer, int M) {
    if (!tap_ || only_class_ >= 0) return HM_OK;
    HM_CUDA(cudaMemcpyAsync(tap_ + ((size_t)layer * tap_rows_ + tap_row0_) * H_, h_, (size_t)M * H_ * 4, cudaMemcpyDeviceToHost, stream_));
    return HM_OK;
}

int Engine::step(const hm_step_entry* entries, int n, float* logits, uint32_t* greedy, float* hidden) {
    if (!set_device()) return fail(HM_ERR_CUDA, "cudaSetDevice failed");
    if (batch_ == 0) return fail(HM_ERR_STATE, "step before kv_alloc");
    if (!entries || n < 1) return fail(HM_ERR_INVALID, "step: bad arguments");
    size_t rows = 0, wants = 0;
    std::vector<char> seen(batch_, 0);
    std::vector<std::pair<int, long>> need;
    for (int i = 0; i < n; ++i) {
        const hm_step_entry& e = entries[i];
        if (e.seq < 0 || e.seq >= batch_ || seen[e.seq]) return fail(HM_ERR_INVALID, "step: sequence index out of range or named twice");
        seen[e.seq] = 1;
        if (e.n_tokens < 1 || !e.tokens || e.n_want < 0 || (e.n_want > 0 && !e.want)) return fail(HM_ERR_INVALID, "step: bad entry");
        for (int k = 0; k < e.n_tokens; ++k)
            if (e.tokens[k] >= (uint32_t)V_) return fail(HM_ERR_INVALID, "step: token id out of range");
        for (int k = 0; k < e.n_want; ++k)
            if (e.want[k] < 0 || e.want[k] >= e.n_tokens || (k > 0 && e.want[k] <= e.want[k - 1])) return fail(HM_ERR_INVALID, "step: wanted places must ascend within the portion");
        if ((long)len_[e.seq] + e.n_tokens > max_seq_)
            return fail(HM_ERR_KV_FULL, "KV cache full (" + std::to_string(len_[e.seq]) + " + " + std::to_string(e.n_tokens) + " > " + std::to_string(max_seq_) + ")");
        need.push_back({e.seq, (long)len_[e.seq] + e.n_tokens});
        rows += e.n_tokens;
        wants += e.n_want;
    }
    const int prc = ensure_pages(need);
    if (prc) return prc;
    HM_CUDA(cudaStreamSynchronize(stream_));
    // staging: tokens, positions, sequences [rows]; wanted rows (index within their pass) and greedy results [rows]; new lengths [batch]
    if (rows > st_rows_) {
        const size_t cap = std::max<size_t>(rows, 256);
        auto re = [&](auto** p) -> cudaError_t {
            if (*p) cudaFree(*p);
            *p = nullptr;
            return cudaMalloc((void**)p, cap * 4);
        };
        st_rows_ = 0;
        HM_CUDA(re(&st_tokens_));
        HM_CUDA(re(&st_pos_));
        HM_CUDA(re(&st_seq_));
        HM_CUDA(re(&st_want_));
        HM_CUDA(re(&st_next_));
        if (st_pin_) cudaFreeHost(st_pin_);
        st_pin_ = nullptr;
        HM_CUDA(cudaMallocHost(&st_pin_, (5 * cap + 2 * (size_t)batch_) * 4));
        st_rows_ = cap;
    }
    uint32_t *p_tok = st_pin_, *p_pos = p_tok + st_rows_, *p_seq = p_pos + st_rows_, *p_want = p_seq + st_rows_, *p_next = p_want + st_rows_, *p_len = p_next + st_rows_;
    const int chunk = std::min(TC_ROWS, scratch_rows_);
    std::vector<int> pass_wants((rows + chunk - 1) / chunk, 0), pass_longest(pass_wants.size(), 0);
    size_t r = 0, q = 0;
    for (int i = 0; i < n; ++i) {
        const hm_step_entry& e = entries[i];
        int w = 0;
        for (int k = 0; k < e.n_tokens; ++k, ++r) {
            p_tok[r] = e.tokens[k];
            p_pos[r] = (uint32_t)(len_[e.seq] + k);
            p_seq[r] = (uint32_t)e.seq;
            pass_longest[r / chunk] = std::max(pass_longest[r / chunk], len_[e.seq] + k + 1);
            if (w < e.n_want && e.want[w] == k) {
                p_want[q++] = (uint32_t)(r % chunk);
                pass_wants[r / chunk]++;
                ++w;
            }
        }
        p_len[2 * i] = (uint32_t)(len_[e.seq] + e.n_tokens);
    }
    HM_CUDA(cudaMemcpyAsync(st_tokens_, p_tok, rows * 4, cudaMemcpyHostToDevice, stream_));
    HM_CUDA(cudaMemcpyAsync(st_pos_, p_pos, rows * 4, cudaMemcpyHostToDevice, stream_));
    HM_CUDA(cudaMemcpyAsync(st_seq_, p_seq, rows * 4, cudaMemcpyHostToDevice, stream_));
    if (wants) HM_CUDA(cudaMemcpyAsync(st_want_, p_want, wants * 4, cudaMemcpyHostToDevice, stream_));
    float* land = logits && wants ? logits_landing(logits, wants * V_ * 4) : nullptr;
    int launches = 0, rc = HM_OK;
    size_t done = 0;
    tap_ = hidden;
    tap_rows_ = rows;
    for (size_t c0 = 0, pass = 0; c0 < rows && rc == HM_OK; c0 += chunk, ++pass) {
        const int mc = (int)std::min<size_t>(chunk, rows - c0), nw = logits || greedy ? pass_wants[pass] : 0;
        tap_row0_ = c0;
        pass_longest_ = pass_longest[pass];
        pass_runs_.clear();
        for (int m = 0; m < mc; ++m) {  // a sequence's tokens are consecutive, so its rows within the pass are one run
            if (m > 0 && p_seq[c0 + m] == p_seq[c0 + m - 1]) pass_runs_.back().second++;
            else pass_runs_.push_back({m, 1});
        }
        lm_pick_ = nw ? st_want_ + done : nullptr;
        rc = enqueue_pass(mc, st_tokens_ + c0, st_pos_ + c0, st_seq_ + c0, 0, nw, false, st_next_ + done, nullptr, nullptr, nullptr, &launches);
        if (rc == HM_OK && nw && logits) {
            const cudaError_t ce = cudaMemcpyAsync(land + done * V_, logits_, (size_t)nw * V_ * 4, cudaMemcpyDeviceToHost, stream_);
            if (ce != cudaSuccess) rc = cuda_fail(ce, "logits copy");
        }
        done += nw;
    }
    pass_runs_.clear();
    tap_ = nullptr;
    lm_pick_ = nullptr;
    if (rc) return rc;
    for (int i = 0; i < n; ++i) {
        const int seq = entries[i].seq;
        HM_CUDA(cudaMemcpyAsync(pos_dev_ + seq, p_len + 2 * i, 4, cudaMemcpyHostToDevice, stream_));
        // what follows a prompt's portion counts as generated for the sampler's penalties
        if (entries[i].n_tokens > 1 || len_[seq] == 0) HM_CUDA(cudaMemcpyAsync(smp_gen_start_ + seq, p_len + 2 * i, 4, cudaMemcpyHostToDevice, stream_));
    }
    if (greedy && wants) HM_CUDA(cudaMemcpyAsync(p_next, st_next_, wants * 4, cudaMemcpyDeviceToHost, stream_));
    if (int qrc = queue_error_copy()) return qrc;
    HM_CUDA(cudaStreamSynchronize(stream_));
    rc = check_device_error();
    if (rc) return rc;
    if (land && land != logits) std::memcpy(logits, land, wants * V_ * 4);
    if (greedy && wants) std::memcpy(greedy, p_next, wants * 4);
    for (int i = 0; i < n; ++i) {
        const int seq = entries[i].seq;
        if (entries[i].n_tokens > 1 || len_[seq] == 0) gen_start_[seq] = len_[seq] + entries[i].n_tokens;
        len_[seq] += entries[i].n_tokens;
    }
    return HM_OK;
}

}  // namespace hm
