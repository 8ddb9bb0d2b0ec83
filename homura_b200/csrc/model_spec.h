// What a checkpoint's config.json describes, in the engine's terms.
//
// Most designs are uniform stacks that hm_config describes completely (Qwen2 / Qwen3 / Llama: grouped-query attention with
// rotation, SwiGLU).  Designs that list their layers one by one fill `layers`; the table in model_spec.cpp maps the
// "architecture" key to the function that reads such a config.
#pragma once
#include <string>
#include <vector>

#include "../../include/homura_b200.h"
#include "loaders.h"

namespace hm {

// MIX_PARALLEL: grouped-query attention and linear attention side by side; MIX_LINEAR: linear attention alone
enum MixerKind { MIX_GQA = 0, MIX_LATENT = 1, MIX_PARALLEL = 2, MIX_LINEAR = 3 };
// Linear attention: a decay per key channel out of a latent; a fixed decay per head; a decay per key channel and the delta rule
enum LinearKind { LIN_GATED = 0, LIN_RETENTION = 1, LIN_DELTA = 2 };
enum MlpKind { MLP_NONE = 0, MLP_SWIGLU = 1, MLP_SQRELU = 2, MLP_MOE = 3, MLP_GLU = 4 };
// RMS norm of queries and keys: none, every head by itself (one weight vector of `dim`), the whole projection at once, every head by
// itself after its rotation and without a weight, the same by the sum of squares instead of their mean
enum QkNorm { QKN_NONE = 0, QKN_HEAD = 1, QKN_ALL = 2, QKN_UNIT = 3, QKN_SUM = 4 };
// Sigmoid gates on an attention's result: none, one per element, one per head
enum OutGate { GATE_NONE = 0, GATE_ELEM = 1, GATE_HEAD = 2 };
// Activations of gated feed-forwards: act(gate) * up
enum GluAct { GLU_CLAMPED = 0, GLU_SILU = 1, GLU_GELU = 2 };

// Rotation of the first `dims` elements of a head: pair i turns by base^(-2 i / dims) per position; `scaled`: wavelengths above
// original / low turn `factor` times slower, those below original / high as they are, with a ramp in between.
struct RotSpec {
    int dims = 0;  // 0: no rotation
    double base = 0;
    bool scaled = false;
    double factor = 1, low = 1, high = 1, original = 1;
};
// Turns (of 2 pi) per position of every pair.
std::vector<double> rotation_turns(const RotSpec& r);

struct LayerSpec {
    int mixer = MIX_GQA;
    // MIX_LATENT: heads of dim query / key and vdim value elements over latents of kv_rank elements
    int heads = 0, dim = 0, vdim = 0, kv_rank = 0;
    int q_rank = 0;        // > 0: queries go through a latent of their own
    int rot_dim = 0;       // rotated elements behind the dim unrotated ones; one rotated key part for all heads is cached behind the latent
    int kv_from = -1;  // layer whose cached latents this one reads (-1: its own)
    float scale = 1.f;
    // MIX_GQA (listed): heads query heads of dim over kv_heads key heads of dim and value heads of vdim
    int kv_heads = 0;
    int qk_norm = QKN_NONE;
    float temp_coef = 0.f;  // queries times 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1); temp_every 0: not
    int temp_every = 0;
    double bias_reach = 0;  // > 0: learned bias by distance, logarithmic steps up to this many tokens back
    bool v_mix = false;     // values are blended with those of layer v_first (which keeps its own)
    int v_first = -1;
    int window = 0;         // > 0: a token sees itself and the window - 1 tokens in front of it,
    int keep_first = 0;     // and the first keep_first tokens
    int chunk = 0;          // > 0: a token sees the tokens of its own chunk of so many, counted from the sequence's start
    bool tied_values = false;  // values are the keys as they are before their rotation
    bool talking = false;   // scores times a temperature per head, then mixed over the heads by a matrix
    bool sink = false;      // one more score per head in the softmax, without a value
    int out_gate = GATE_NONE;
    bool qkv_bias = false;
    int conv = 0;           // taps of a causal convolution per channel of queries, keys and values; 0: none
    RotSpec rot;            // also that of MIX_LATENT
    // MIX_PARALLEL: beside the attention above, gated linear attention with a decay per key channel
    int lin_kind = LIN_GATED;
    int lin_heads = 0, lin_dim = 0, lin_vdim = 0;
    int lin_kv_heads = 0;   // LIN_DELTA: heads of queries and keys
    int lin_conv = 0;       // LIN_DELTA: taps of a causal convolution per channel of queries, keys and values
    std::vector<float> lin_decay;  // LIN_RETENTION: per head
    float lin_tau = 1.f;
    int decay_rank = 0;     // from the tensors
    int gate_rank = 0;      // LIN_DELTA: latent of the output gate, from the tensors
    float left_scale = 1.f, right_scale = 1.f;
    int mlp = MLP_NONE;
    int ff = 0;             // of one expert with MLP_MOE
    int act = GLU_CLAMPED;  // MLP_MOE, MLP_GLU
    float router_scale = 1.f;
    int shared_ff = 0;      // MLP_MOE: > 0: an expert that every token runs, times a sigmoid
    // MLP_MOE: `top` of experts + identity router outputs; the identity ones pass their input on
    int experts = 0, identity = 0, top = 0;
    float limit = 0.f;      // GLU_CLAMPED: clamp of gate (above) and up (both sides)
    bool mlp_bias = false;
    bool linear() const { return mixer == MIX_PARALLEL || mixer == MIX_LINEAR; }
    bool paged_kv() const { return mixer == MIX_GQA || mixer == MIX_PARALLEL; }  // caches keys and values
    int lin_channels() const { return 2 * lin_kv_heads * lin_dim + lin_heads * lin_vdim; }  // LIN_DELTA: queries, keys and values
    int latent_rank() const { return kv_rank + rot_dim; }      // elements of a cached latent row
    int q_stride() const { return (dim + rot_dim + 7) / 8 * 8; }  // q_rank: a head's queries, rotated pairs first
};

struct ModelSpec {
    hm_config cfg{};          // sizes every design has; the largest over the layers where they differ
    std::string arch;         // "" for the uniform stacks
    std::vector<LayerSpec> layers;  // empty for the uniform stacks
    int norm_groups = 1;      // runs of the width that a norm divides by their own root mean square
    bool token_shift = false; // the mixer reads a blend of a token's normalised row and its predecessor's
    bool layer_scale = false; // mixer and MLP results are multiplied element by element before they join the residual
    bool post_norm = false;   // mixer and MLP read the residual itself; their results are normalised, times residual_mult, before they join it
    float residual_mult = 1.f;
    bool sin_pos = false;     // sinusoidal position vectors are added to the embedding
    bool parallel = false;    // mixer and MLP read one norm of the residual and are added to it together
    bool sandwich = false;    // mixer and MLP read a layer norm of the residual and give back through another one
    float logit_scale = 1.f;
    bool norm_offset = false; // norm weights are stored as their distance from one
    float embed_scale = 1.f;
    // a second embedding by (previous token * mul_prev + token * mul_cur) mod buckets, row `buckets` for a sequence's first token
    long long bigram_buckets = 0, bigram_prev = 0, bigram_cur = 0;
    float softcap = 0.f;      // > 0: logits are softcap * tanh(logits / softcap)
    bool listed() const { return !layers.empty(); }
};

// config.json text -> spec.  An "architecture" of the table goes to its reader, anything else to the uniform stacks.
bool parse_model_spec(const char* text, size_t len, ModelSpec* out, std::string* err);
bool parse_model_spec_file(const std::string& path, ModelSpec* out, std::string* err);
// The layer list as JSON (hm_checkpoint_info); "[]" for the uniform stacks.
std::string layers_json(const ModelSpec& spec);

}  // namespace hm
