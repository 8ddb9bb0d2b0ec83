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

enum MixerKind { MIX_GQA = 0, MIX_LATENT = 1 };
enum MlpKind { MLP_NONE = 0, MLP_SWIGLU = 1, MLP_SQRELU = 2, MLP_MOE = 3 };
// RMS norm of queries and keys: none, every head by itself (one weight vector of `dim`), the whole projection at once
enum QkNorm { QKN_NONE = 0, QKN_HEAD = 1, QKN_ALL = 2 };

struct LayerSpec {
    int mixer = MIX_GQA;
    // MIX_LATENT: heads of dim query / key and vdim value elements over latents of kv_rank elements
    int heads = 0, dim = 0, vdim = 0, kv_rank = 0;
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
    int mlp = MLP_NONE;
    int ff = 0;             // of one expert with MLP_MOE
    // MLP_MOE: `top` of experts + identity router outputs; the identity ones pass their input on
    int experts = 0, identity = 0, top = 0;
    float limit = 0.f;      // clamp of the experts' gate (above) and up (both sides)
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
    bool listed() const { return !layers.empty(); }
};

// config.json text -> spec.  An "architecture" of the table goes to its reader, anything else to the uniform stacks.
bool parse_model_spec(const char* text, size_t len, ModelSpec* out, std::string* err);
bool parse_model_spec_file(const std::string& path, ModelSpec* out, std::string* err);
// The layer list as JSON (hm_checkpoint_info); "[]" for the uniform stacks.
std::string layers_json(const ModelSpec& spec);

}  // namespace hm
