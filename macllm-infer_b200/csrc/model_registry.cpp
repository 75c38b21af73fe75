// See model_registry.h.
#include "model_registry.h"

namespace mk {

namespace {
std::vector<ModelFormat>& formats() {
    static std::vector<ModelFormat> all;
    return all;
}
}  // namespace

RegisterModelFormat::RegisterModelFormat(ModelFormat f) { formats().push_back(std::move(f)); }

std::unique_ptr<PagedLm> load_model(const std::string& path, const ModelConfig& cfg) {
    std::string known;
    for (const ModelFormat& f : formats()) {
        if (f.matches(path)) return f.load(path, cfg);
        known += (known.empty() ? "" : ", ") + f.name;
    }
    throw std::runtime_error("`" + path + "` is no checkpoint of a known format (" + known + ")");
}

}  // namespace mk
