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
enum MlpKind { MLP_NONE = 0, MLP_SWIGLU = 1, MLP_SQRELU = 2 };

struct LayerSpec {
    int mixer = MIX_GQA;
    // MIX_LATENT: heads of dim query / key and vdim value elements over latents of kv_rank elements
    int heads = 0, dim = 0, vdim = 0, kv_rank = 0;
    int kv_from = -1;  // layer whose cached latents this one reads (-1: its own)
    float scale = 1.f;
    int mlp = MLP_NONE;
    int ff = 0;
};

struct ModelSpec {
    hm_config cfg{};          // sizes every design has; the largest over the layers where they differ
    std::string arch;         // "" for the uniform stacks
    std::vector<LayerSpec> layers;  // empty for the uniform stacks
    int norm_groups = 1;      // runs of the width that a norm divides by their own root mean square
    bool token_shift = false; // the mixer reads a blend of a token's normalised row and its predecessor's
    bool layer_scale = false; // mixer and MLP results are multiplied element by element before they join the residual
    bool listed() const { return !layers.empty(); }
};

// config.json text -> spec.  An "architecture" of the table goes to its reader, anything else to the uniform stacks.
bool parse_model_spec(const char* text, size_t len, ModelSpec* out, std::string* err);
bool parse_model_spec_file(const std::string& path, ModelSpec* out, std::string* err);
// The layer list as JSON (hm_checkpoint_info); "[]" for the uniform stacks.
std::string layers_json(const ModelSpec& spec);

}  // namespace hm
