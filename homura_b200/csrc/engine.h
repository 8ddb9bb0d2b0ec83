// Device-resident decode engine: weights, paged KV cache, the decode step as a CUDA graph.
//
// Takes the place of HfModel + ExecutionPlan::run_kv on the decode path
// (src/hf/model.rs:37-267, src/runtime.rs:1580-1892): instead of routing host Buffers
// between ~5 compiled kernels per layer, the step is a fixed chain of fused kernels whose
// activations never leave HBM, captured once and replayed per token.
#pragma once
#include <cuda_runtime.h>

#include <string>
#include <vector>

#include "../../include/homura_b200.h"
#include "common.cuh"
#include "gla.h"
#include "gqa_attn.h"
#include "latent_attn.h"
#include "moe.h"
#include "model_spec.h"
#include "recur.h"
#include "sampler.h"
#include "side.h"

namespace hm {

struct TcArgs;

struct LinearW {
    int K = 0, N = 0;        // N = output count of the (possibly fused) projection
    int kind = -1;           // HM_BF16 (slab layout) | HM_Q8_0 | HM_Q4_0 (split scales + codes)
    uint16_t* slabs = nullptr;
    uint16_t* tc = nullptr;  // second copy in the tensor-core tile layout (gemm_tc.h), used for passes over more than 8 rows
    uint16_t* scales = nullptr;
    uint8_t* codes = nullptr;
    uint8_t* kq_data = nullptr;       // K-quants (kind HM_Q4_K stands for the family): tiled super-blocks, kquant.h
    uint8_t* kq_tile_type = nullptr;  // per 32-row tile: 1 = Q4_K, 2 = Q6_K
    size_t kq_bytes = 0;              // GGUF bytes loaded into it (what a step streams)
    int kq_part_type = -1;            // type of the part loaded last (gate and up must agree: they share tiles)
    bool kq_has_q6 = false;           // some tile is Q6_K: passes over more than 8 rows keep the 8-row launches (the row-block kernel is Q4_K only)
    int loaded_parts = 0;
    // grouped (block-diagonal) projection: K inputs and group_n outputs per group, every group in group_slabs 128-column slabs of its own
    int groups = 0, group_n = 0, group_slabs = 0;
    int columns() const { return groups ? groups * group_slabs * SLAB : N; }  // output columns counting the padding between groups
    bool rope_rows = false;  // quantised fused QKV: q and k rows stored in rotation-pair tiles (rope_tile_row), the projection's epilogue rotates
    size_t bytes() const;
};

struct LayerW {
    float* in_ln = nullptr;
    float* post_ln = nullptr;
    float* qkv_bias = nullptr;  // fused [q_dim + 2 kv_dim]
    float* q_norm = nullptr;
    float* k_norm = nullptr;
    LinearW qkv, o, gu, down;  // listed designs: gu is the up projection alone, qkv is empty
    // listed designs (ModelSpec::layers)
    float* shift = nullptr;              // token shift [H]
    float *ls1 = nullptr, *ls2 = nullptr;  // layer scales [H]
    float* latent_norm = nullptr;        // [kv_rank]
    LinearW in;                          // queries, output gate and (unless another layer's latents are used) latents, parts padded to 128 columns
    LinearW kup, vup;                    // per head: query -> latent space, latent space -> values
    // listed grouped-query attention: `in` is queries, keys and values without padding
    float* v_mix = nullptr;              // share of the first such layer's values
    float* rel = nullptr;                // distance bias [heads][reach + 1]
    int reach = 0;
    // mixture of experts
    uint16_t* router = nullptr;          // [experts + identity][H] bf16
    float* correction = nullptr;
    uint16_t *exp_gu = nullptr, *exp_down = nullptr;  // all experts' tile images (moe.h)
    std::vector<uint8_t> exp_seen;       // per expert: bits of the parts loaded
    // listed designs with parallel sublayers: `in` is everything that reads the norm, `o` everything that joins the residual (besides
    // the chosen experts), see ParallelColumns
    std::vector<std::string> seen;       // tensors loaded
    float* in_bias = nullptr;            // [columns of `in`]
    float* sink = nullptr;               // [heads]
    float* conv_w = nullptr;             // [query, key and value channels][taps]
    float *lin_norm = nullptr, *lin_up = nullptr, *lin_bias = nullptr;  // linear attention: result norm, decay up-projection [heads][rank][dim], its bias
    LinearW uq;                          // queries out of their latent
    // listed designs with sublayers between two norms: `in` is everything that the mixer reads off its normed input
    float *norm1b = nullptr, *norm2b = nullptr;  // norms behind mixer and MLP
    float *left_out = nullptr, *right_out = nullptr;  // norms of a parallel mixer's two results
    float *talk = nullptr, *temp = nullptr;  // mixing matrix of the heads' scores, temperatures
    float *gu_bias = nullptr, *down_bias = nullptr;
    std::vector<float> gu_bias_host;     // gate and up interleaved as their rows are
    float *lin_conv_w = nullptr, *lin_rate = nullptr, *lin_up_g = nullptr, *lin_decay = nullptr;  // delta rule: convolution, -exp(A_log), gate up-projection; retention: decays
    size_t lin_conv_at = 0;
    struct Pending { std::string name, rest; int dtype; std::vector<int64_t> shape; std::vector<uint8_t> data; };
    std::vector<Pending> pending;        // tensors that came before those that tell their layer's sizes
    double* turns = nullptr;             // rotation, turns per position of every pair
    size_t conv_at = 0, gla_at = 0;      // this layer's part of a sequence's state, in floats
};

// What a projection launch needs beyond the common arguments (enqueue_linear)
struct LinOpt {
    RowNorm gn{};                        // with PRO_GNORM
    SplitRows split{};                   // with PRO_MERGE
    const float* out_scale = nullptr;
    const float* gate = nullptr;
    int ld_gate = 0;
    int group_x = 0;                     // grouped projections: inputs of one group to the next
    int gate_per = 0;                    // EPI_GATE: columns that share a gate
    float limit = 0.f;                   // EPI_GLU
    int glu_n = 0;
    TurnedPairs turn{};
    float softcap = 0.f;
};

// Columns of a parallel layer's input projection (what reads the norm of the residual) and inputs of its output projection (what
// joins the residual).  Parts start at multiples of 8 columns and of 64 inputs; queries, keys and values are contiguous.
struct ParallelColumns {
    int q = 0, k = 0, v = 0, gate = 0, gates = 0;          // attention, its output gates
    int lq = 0, lk = 0, lv = 0, lg = 0, la = 0;            // linear attention, gate, decay latent
    int lb = 0, lgl = 0;                                   // delta rule: step sizes, gate latent
    int dq = 0, dkv = 0;                                   // latents of queries; of keys and values with the rotated part behind
    int router = 0, row_gate = 0, ff_gate = 0, ff_up = 0, ff = 0;  // dense or shared feed-forward
    int n = 0, ld = 0;
    int vals = 0, lin_in = 0, ff_in = 0, k_out = 0;
};

// final argmax folded into the LM-head launch (see GemvArgs::fin_ticket)
struct ArgmaxFold {
    uint32_t *next_tok, *feed_tok;
    int32_t* pos;
    uint32_t* hist;
    int hist_stride;
};

class Engine {
   public:
    // strict_f32: projections on the f32 streaming kernels only (no tensor-core copies of the weights)
    static int create(const ModelSpec& spec, int device, bool strict_f32, Engine** out, std::string* err);
    ~Engine();

    // Shape of a tensor that load_tensor will bring: sizes that only tensors tell must be known before their layer's projections.
    void note_shape(const std::string& name, const std::vector<int64_t>& shape);
    int load_tensor(const char* name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int finalize();

    // pool_tokens 0: every sequence owns pages for max_seq_len tokens; else the sequences share a pool of that many tokens and
    // take pages from it as they grow
    int kv_alloc(int batch, int max_seq_len, int page_tokens, int kv_dtype, long pool_tokens = 0);
    int kv_free_tokens(long* out);
    int latent_view(int seq, int layer, float* out);
    // One batch over several sequences, each bringing any number of tokens
    int step(const hm_step_entry* entries, int n, float* logits, uint32_t* greedy, float* hidden);
    int kv_free();
    int kv_reset(int seq);
    int kv_len(int seq, int* out);
    int kv_append(int seq, int layer, const float* k_rows, const float* v_rows, int n_new, int advance);
    int kv_view(int seq, int layer, float* k_out, float* v_out);

    int prefill(int seq, const int64_t* ids, int n, float* logits, uint32_t* first_token);
    int decode_step(const uint32_t* tokens, float* logits, uint32_t* next_tokens);
    int decode_step_sampled(const uint32_t* tokens, const hm_sampling* s, uint64_t* rng_state, float* logits, uint32_t* next_tokens);
    int decode_greedy_n(const uint32_t* first_tokens, int steps, uint32_t* out_ids);
    int generate(int seq, const int64_t* prompt, int n_prompt, int max_new, const hm_sampling* s, uint32_t* out_ids, int* n_out);
    int time_decode(int warmup, int steps, float* ms_total);
    int profile_decode(int steps, hm_kernel_stat* out, int cap, int* n_out);
    int selftest_expire_wait();

    const hm_config& config() const { return cfg_; }
    const ModelSpec& spec() const { return spec_; }
    uint64_t weight_bytes() const;
    cudaStream_t stream() const { return stream_; }
    int launches_per_step() const { return launches_per_step_; }
    std::string err;

   private:
    Engine() = default;
    int fail(int code, const std::string& msg);
    int cuda_fail(cudaError_t e, const char* what);
    bool set_device();
    int stage(const void* host, size_t nbytes, void** dev);  // temp device copy of a host tensor
    int load_linear(LinearW& L, int K, int N_total, int n_off, int n_part, int interleave_which, int dtype, const void* host, size_t nbytes, int rope_part = 0);
    int load_vec_f32(float** dst, size_t n_total, size_t off, int dtype, const void* host, size_t n, size_t nbytes);
    int ensure_scratch(int rows);
    RopeEpi rope_epi(int layer, const int32_t* row_pos, const int32_t* row_seq, int m0) const;
    // Enqueue one pass over M rows (decode: one row per sequence; prefill: a chunk of one
    // sequence).  lm_row0/lm_rows select the rows that go through the LM head.
    int enqueue_pass(int M, const uint32_t* tokens_dev, const int32_t* row_pos, const int32_t* row_seq, int lm_row0, int lm_rows, bool advance, uint32_t* next_dev, uint32_t* feed_dev, int32_t* pos_dev, uint32_t* hist_dev, int* launches);
    int enqueue_linear(const LinearW& L, int M, const float* x, int ldx, int pro, const float* norm_w, int epi, float* y, int ldy, const float* bias, const float* resid, int layer, const int32_t* row_pos, const int32_t* row_seq, float* amax_val, int32_t* amax_idx, int* launches, const struct ArgmaxFold* fold = nullptr, const LinOpt* opt = nullptr);
    // listed designs (engine_listed.cu)
    int load_listed_tensor(const std::string& name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int load_grouped(LinearW& L, int groups, int K, int group_n, bool src_is_kn, int dtype, const void* host, size_t nbytes);
    int finalize_listed();
    int alloc_listed_scratch(int cap);
    int alloc_listed_cache(int batch, size_t n_pages);
    void free_listed_cache();
    void free_listed();
    // Rows from which a pass's projections run on the tensor cores.  The grouped norms of listed designs cost the streaming kernel
    // more per row, so theirs move over earlier.
    bool tall_rows(int rows) const { return use_tc_ && rows > (spec_.listed() ? 4 : MAX_M); }
    int enqueue_listed_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int next_lm_rows, int* launches);
    // listed grouped-query attention, post-norms, mixtures of experts (engine_gqa.cu)
    int load_gqa_tensor(LayerW& w, const LayerSpec& s, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int load_bias_table(LayerW& w, const LayerSpec& s, int dtype, const int64_t* shape, const void* host, size_t nbytes);
    int load_expert(LayerW& w, const LayerSpec& s, int expert, int part, int dtype, const void* host, size_t nbytes);
    bool load_expert_tensor(LayerW& w, const LayerSpec& s, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes, int* rc);
    int finalize_gqa(const LayerW& w, const LayerSpec& s, const std::string& at);
    int alloc_gqa_scratch();
    void free_gqa_scratch();
    GqaPool gqa_pool(int layer) const;
    RouteOut route_out(bool dense) const;
    double experts_used(const LayerSpec& s, int rows) const;
    ExpertWeights expert_weights(int layer) const;
    uint64_t expert_bytes(int layer, bool gate_up) const;
    int count_experts(int M, const LayerSpec& s);
    int enqueue_gqa_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int next_lm_rows, int* launches);
    // listed designs with parallel sublayers (engine_parallel.cu)
    int load_parallel_tensor(int layer, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int load_inputs(LinearW& L, int k_total, int k_off, int k_part, int N, int dtype, const void* host, size_t nbytes);
    int load_bigram(int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int upload(float** dst, const std::vector<float>& v);
    int finalize_parallel();
    int alloc_parallel_scratch();
    void free_parallel_scratch();
    SideArgs side_args(int l, int M, bool tall, const ParallelColumns& c, const int32_t* row_pos, const int32_t* row_seq) const;
    int enqueue_parallel_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int next_lm_rows, int* launches);
    // listed designs with sublayers between two norms (engine_sandwich.cu)
    int load_sandwich_tensor(int layer, const std::string& name, const std::string& rest, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int load_group(LinearW& L, int groups, int g, int K, int k_part, int group_n, int dtype, const void* host, size_t nbytes);
    int finalize_sandwich();
    int alloc_sandwich_scratch();
    int enqueue_sandwich(int M, bool tall, const LayerW* joined, const float* post_w, const float* next_w, int* launches);
    SideArgs sandwich_side_args(int l, int M, const int32_t* row_pos, const int32_t* row_seq) const;
    RecurArgs recur_args(int l, int M, bool tall, const int32_t* row_pos, const int32_t* row_seq) const;
    int enqueue_sandwich_layer(int l, int M, const int32_t* row_pos, const int32_t* row_seq, int lm_rows, int* launches);
    int enqueue_sandwich_logits(const float* x, int rows, bool normed, float* dst, const struct ArgmaxFold& fold, int* launches);
    bool final_norm_fits(int M, int lm_rows) const { return lm_rows == M && !lm_pick_; }
    // shared by the listed designs
    int load_key_up(LayerW& w, const LayerSpec& s, const std::string& name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    int load_value_up(LayerW& w, const LayerSpec& s, const std::string& name, int dtype, const int64_t* shape, int ndim, const void* host, size_t nbytes);
    GqaRuns pass_runs(int M, int* longest) const;
    GqaAttnArgs gqa_attn_args(int l, int M, bool tall, const int32_t* row_pos, const int32_t* row_seq) const;
    int enqueue_latent_attn(int l, int M, bool tall, const int32_t* row_pos, const int32_t* row_seq, int* launches);
    // x: the rows that the experts read (few rows); resid: added to the result (few rows) or null.  With many rows `parts` partial results in sub_.
    int enqueue_experts(int l, int M, bool tall, const float* x, const float* resid, float* y, int* parts, int* launches);
    int enqueue_listed_logits(const float* x, int rows, float* dst, const struct ArgmaxFold& fold, int* launches);
    int enqueue_tc(const LinearW& L, int M, const unsigned char* xp, int epi, float* y, int ldy, TcArgs& a, int* launches);
    LatentPool latent_pool(int layer) const;
    // The per-sequence state that is not addressed by position (token shift): copies of one sequence's, for generation loops
    // that run ahead of the host, and the way back from a run that went too far.
    int save_state(int seq);
    int rewind(int seq, int len, const std::vector<uint32_t>& fed);
    // pages
    int ensure_pages(const std::vector<std::pair<int, long>>& need);  // (sequence, tokens it will hold)
    int ensure_pages_all(int more);
    void release_pages(int seq);
    template <typename F>
    void each_linear(F f) {
        for (auto& l : layers_)
            for (LinearW* w : {&l.qkv, &l.o, &l.gu, &l.down, &l.in, &l.kup, &l.vup, &l.uq}) f(*w);
        f(lm_head_);
    }
    // RMSNorm handed from one tensor-core GEMM to the next without a packing launch (see TcArgs)
    struct TcFuse {
        const float* ss_in = nullptr;   // consumer: partial sums of squares of the rows of `prepacked`
        int ss_parts = 0;
        unsigned char* xp_next = nullptr;  // producer: activation image of the next GEMM, scaled by next_norm_w
        const float* next_norm_w = nullptr;
        float* ss_out = nullptr;
    };
    int enqueue_linear_tc(const LinearW& L, int M, const float* x, int ldx, const float* norm_w, int epi, float* y, int ldy, const float* bias, const float* resid, int layer, const int32_t* row_pos, const int32_t* row_seq, int* launches,
                          const unsigned char* prepacked = nullptr, unsigned char* pack_out = nullptr, const TcFuse* fuse = nullptr);
    int capture_decode_graph();
    int ensure_host_logits_graph();
    int ensure_sampler_scratch();
    SamplerArgs sampler_args(const hm_sampling& s) const;
    int launch_step();        // replay the captured decode graph
    int queue_error_copy();    // device error word -> pinned host word, on the engine's stream
    int check_device_error();  // after the synchronisation that follows queue_error_copy()
    void prof_mark(int cls);

    ModelSpec spec_;
    hm_config cfg_{};
    int device_ = 0, sm_count_ = 148;
    int H_ = 0, I_ = 0, heads_ = 0, kvh_ = 0, hd_ = 0, qdim_ = 0, kvdim_ = 0, L_ = 0, V_ = 0;
    bool finalized_ = false, quant_ = false, pdl_ = true;
    bool use_clusters_ = true;  // split reductions through thread-block clusters / DSMEM (HM_NO_CLUSTER=1: global scratch + tickets)
    int max_cluster_ = 8;
    bool use_prefetch_ = true;  // decode kernels pull the weights of the kernel two launches ahead into the L2
    const void* pf_ptr_ = nullptr;  // prefetch target handed to the next projection launch
    unsigned long long pf_bytes_ = 0;
    bool use_tc_ = true;  // bf16 models: passes over more than 8 rows run the tcgen05 GEMM (HM_NO_TC=1: 8-row groups of the streaming kernel)
    cudaStream_t stream_ = nullptr;

    // weights
    void* embed_ = nullptr;  // [V,H] bf16 (embed_dtype_ == HM_BF16) or f32
    int embed_dtype_ = -1;
    float* final_norm_ = nullptr;
    std::vector<LayerW> layers_;
    LinearW lm_head_;
    float *rope_cos_ = nullptr, *rope_sin_ = nullptr;

    // activations / scratch for up to scratch_rows_ rows
    int scratch_rows_ = 0;
    float *h_ = nullptr, *q_ = nullptr, *attn_ = nullptr, *act_ = nullptr, *qkv_raw_ = nullptr, *gu_raw_ = nullptr, *logits_ = nullptr;
    unsigned char* xpack_ = nullptr;  // packed activations of one tensor-core projection (gemm_tc.h)
    unsigned char *xpack_attn_ = nullptr, *xpack_act_ = nullptr;  // written directly by the attention kernel / the SwiGLU epilogue
    unsigned char *xpack_h_ = nullptr, *xpack_h2_ = nullptr;      // written by the down / O epilogues: (hidden * next norm weight) for the next QKV or LM head / gate-up GEMM
    float *ss_h_ = nullptr, *ss_h2_ = nullptr;                    // [H/128][64] partial sums of squares of those rows
    uint32_t* qrows_img_ = nullptr;  // Q8_0 / Q4_0 models: digit planes of the up to 64 rows a projection launch multiplies (launch_gemm_quant)
    float* qrows_bs_ = nullptr;      // their block scales
    int qrows_k_ = 0;                // widest projection input the two buffers hold
    int8_t* kqrows_codes_ = nullptr;  // K-quant models: Q8_K codes of the up to 64 rows a projection launch multiplies (launch_gemm_q4k)
    float* kqrows_actd_ = nullptr;    // their block scales
    size_t xpack_bytes_ = 0;
    float* amax_val_ = nullptr;
    int32_t* amax_idx_ = nullptr;
    float* partial_ = nullptr;
    size_t partial_floats_ = 0;
    unsigned int* tickets_ = nullptr;
    float *att_acc_ = nullptr, *att_ml_ = nullptr;
    unsigned int* att_tickets_ = nullptr;
    int att_nsplit_ = 1;
    bool att_cluster_ = true;
    int* err_flag_ = nullptr;
    unsigned int* fin_ticket_ = nullptr;  // ticket of the LM head's folded argmax

    // listed designs
    float *mix_raw_ = nullptr, *qlat_ = nullptr, *ctx_ = nullptr;  // input projection, queries in latent space, attention result in latent space
    unsigned char *xpack_q_ = nullptr, *xpack_ctx_ = nullptr;      // their tensor-core images, one per head
    float *lat_acc_ = nullptr, *lat_ml_ = nullptr;                 // split attention
    size_t lat_acc_floats_ = 0, lat_ml_floats_ = 0;
    std::vector<void*> lat_pool_;  // per layer, null for layers that read another's
    float *shift_state_ = nullptr, *shift_saved_ = nullptr;  // [layers][sequences][SHIFT_RING][H]; [layers][SHIFT_RING][H]
    // State of a sequence that is not addressed by position: short convolutions and linear attention of all layers, one row per
    // sequence; [state_floats_] for the copy that generation loops take
    float *state_ = nullptr, *state_saved_ = nullptr;
    size_t state_floats_ = 0;
    uint16_t* bigram_ = nullptr;     // second embedding table
    float* normed_ = nullptr;        // normalised input of a layer, for experts that read rows
    float* cat_ = nullptr;           // inputs of a parallel layer's output projection,
    unsigned char *xpack_cat_ = nullptr, *xpack_cq_ = nullptr;  // their image; that of the queries' latents
    int cat_ld_ = 0;
    float* lin_rows_ = nullptr;      // rows of a pass that are prepared for a recurrence
    double* turns_ = nullptr;        // sinusoidal positions: turns per position of every pair of elements
    float* sub_ = nullptr;           // what a sublayer gave back, before its norm
    float* v_first_ = nullptr;       // values of the layer that the others blend in
    int32_t* rt_ids_ = nullptr;      // router's choice (RouteOut)
    float *rt_weights_ = nullptr, *rt_identity_ = nullptr, *rt_dense_ = nullptr;
    uint32_t* rt_mask_ = nullptr;
    float* exp_act_ = nullptr;       // activations of the chosen experts: few rows,
    unsigned char* exp_img_ = nullptr;  // or an image per expert
    int sub_parts_ = 1;              // partial results sub_ has room for
    std::vector<int>* experts_seen_ = nullptr;  // profile: experts used per layer of the pass being enqueued
    std::vector<int> experts_read_;  // their counts of the last profiled step
    int32_t* seq_iota_ = nullptr;    // 0, 1, 2, ...: the sequence of every row of a decode step
    int pass_nsplit_ = 1;            // splits the attention of the layer being enqueued left for the next projection to combine
    int pass_longest_ = 0;           // longest context of the pass being enqueued (splits of the attention)
    std::vector<std::pair<int, int>> pass_runs_;  // that pass's runs: first row, rows; empty: a run per row
    // portions (step)
    float* hsel_ = nullptr;              // rows whose logits are wanted
    const int32_t* lm_pick_ = nullptr;   // their indices within the pass being enqueued (null: lm_row0 ..)
    size_t lm_dst_row_ = 0;              // first row of logits_ the pass writes
    uint32_t *st_tokens_ = nullptr, *st_next_ = nullptr;
    int32_t *st_pos_ = nullptr, *st_seq_ = nullptr, *st_want_ = nullptr;
    uint32_t* st_pin_ = nullptr;
    size_t st_rows_ = 0;
    float* tap_ = nullptr;               // host: residual stream after every layer, [layers][tap_rows_][H]
    size_t tap_rows_ = 0, tap_row0_ = 0;
    int tap(int layer, int M);

    // pages
    bool pooled_ = false;
    std::vector<int32_t> free_pages_;
    std::vector<std::vector<int32_t>> seq_pages_;

    // KV cache
    int batch_ = 0, max_seq_ = 0, page_tokens_ = 16, max_pages_ = 0;
    bool kv_bf16_ = false;
    std::vector<void*> k_pool_, v_pool_;
    int32_t* page_table_ = nullptr;
    int32_t* pos_dev_ = nullptr;      // [batch] current length = position of the next token
    uint32_t* tokens_dev_ = nullptr;  // [batch] input token of the next decode step
    uint32_t* next_dev_ = nullptr;    // [batch] argmax of the last step
    uint32_t* hist_dev_ = nullptr;    // [batch][max_seq+1] token history by position
    std::vector<int> len_;            // host mirror of pos_dev_
    // prefill staging (device), capacity max_seq_
    uint32_t* pf_tokens_ = nullptr;
    int32_t *pf_pos_ = nullptr, *pf_seq_ = nullptr;
    // pinned host staging
    uint32_t* pin_u32_ = nullptr;
    size_t pin_u32_cap_ = 0;
    float* pin_logits_ = nullptr;      // mapped pinned buffer: landing place of logits on their way to pageable memory
    float* pin_logits_dev_ = nullptr;  // the same buffer as the device addresses it
    size_t pin_logits_bytes_ = 0;
    bool alloc_pin_logits(size_t bytes);
    float* logits_landing(float* user, size_t bytes);
    // decode graph whose LM head stores the logits straight into pin_logits_ (see ensure_host_logits_graph)
    cudaGraph_t graph_host_ = nullptr;
    cudaGraphExec_t graph_exec_host_ = nullptr;
    bool host_graph_tried_ = false;
    float* lm_out_ = nullptr;  // LM-head destination override while that graph is being captured
    void drop_host_logits_graph();

    cudaGraph_t graph_ = nullptr;
    cudaGraphExec_t graph_exec_ = nullptr;
    int launches_per_step_ = 0;

    int only_class_ = -1;
    bool lm_folds_argmax_ = false;  // the LM-head launch of the last enqueued pass also did the final argmax
    unsigned long long* gemv_trace_ = nullptr;  // builds with -DHM_PHASE_TRACE and HM_GEMV_TRACE=1: [512][16] timestamps, one row per launch of a pass

    // device-side sampler scratch (sampler.cu), allocated on first sampled generation
    float* smp_scaled_ = nullptr;
    int* smp_count_ = nullptr;
    unsigned long long* smp_rng_ = nullptr;
    int32_t* smp_gen_start_ = nullptr;
    int* smp_overflow_ = nullptr;
    std::vector<int> gen_start_;  // host mirror of smp_gen_start_
};

}  // namespace hm
