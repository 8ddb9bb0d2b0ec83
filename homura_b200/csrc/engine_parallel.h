// Shared by the engine's translation units.
#pragma once
#include "engine.h"

namespace hm {
ParallelColumns parallel_columns(const LayerSpec& s);
ParallelColumns sandwich_columns(const LayerSpec& s);
}  // namespace hm
