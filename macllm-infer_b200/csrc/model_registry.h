// The registry of checkpoint formats and of the architectures a format serves.  A translation unit that implements one
// registers it from a static object, so which of them a build carries is decided by what is linked into it.
#pragma once
#include "model_config.h"
#include "paged_lm.h"
#include <functional>
#include <memory>
#include <string>
#include <vector>

namespace mk {

struct ModelFormat {
    std::string name;
    std::function<bool(const std::string& path)> matches;
    std::function<std::unique_ptr<PagedLm>(const std::string& path, const ModelConfig& cfg)> load;
};

struct RegisterModelFormat {
    explicit RegisterModelFormat(ModelFormat f);
};

// Loads the checkpoint with the first registered format that recognises it.
std::unique_ptr<PagedLm> load_model(const std::string& path, const ModelConfig& cfg);

}  // namespace mk
