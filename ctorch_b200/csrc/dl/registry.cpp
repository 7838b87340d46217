// Registry of model designs and loading of a model folder (config.json + model.safetensors).
#include "dl/hybrid.h"
#include "dl/internal.h"

#include <fstream>
#include <sstream>
#include <stdexcept>

namespace dl::models {

namespace {

using Factory = std::shared_ptr<nn::UnaryModule> (*)(const Json&, TensorOptions);

using nn::MixerKind;

constexpr nn::MixerDesign kHybridMixers[] = {{"mamba2", MixerKind::state_space}, {"latent_attention", MixerKind::latent}};
using nn::OutputGate;

constexpr nn::MixerDesign kParallelMixers[] = {{"attention", MixerKind::attention, {.norm = B200_HEAD_NORM_PROJECTION, .gate = OutputGate::head}}};
constexpr nn::MixerDesign kSandwichMixers[] = {
    {"attention", MixerKind::attention, {.norm = B200_HEAD_NORM_NONE, .rotate_pairs = true, .bias = true, .keys_as_values = true, .gate = OutputGate::head, .sink = nn::Sink::zero}},
    {"attention_2", MixerKind::attention, {.norm = B200_HEAD_NORM_HEAD, .rotate_pairs = true, .sink = nn::Sink::learned}},
    {"parallel", MixerKind::side_by_side, {.norm = B200_HEAD_NORM_PROJECTION, .gate = OutputGate::head, .sink = nn::Sink::learned}},
};
constexpr nn::MixerDesign kPostNormMixers[] = {
    {"attention", MixerKind::attention, {.norm = B200_HEAD_NORM_PROJECTION, .gate = OutputGate::value, .mask = nn::AttentionMask::window, .norm_values = true}},
    {"attention_2", MixerKind::attention, {.norm = B200_HEAD_NORM_HEAD, .mask = nn::AttentionMask::window, .head_weights = true, .talk = true}},
    {"delta", MixerKind::delta},
};

std::shared_ptr<nn::UnaryModule> hybrid(const Json& config, TensorOptions options) {
    return std::make_shared<nn::HybridDecoder>(
        config, nn::DecoderDesign{nn::NormKind::dynamic_tanh, nn::LoopEntry::step, nn::LayerForm::sequential, true, kHybridMixers, std::nullopt}, options);
}
std::shared_ptr<nn::UnaryModule> parallel(const Json& config, TensorOptions options) {
    return std::make_shared<nn::HybridDecoder>(
        config, nn::DecoderDesign{nn::NormKind::rms, nn::LoopEntry::joined, nn::LayerForm::parallel, false, kParallelMixers, nn::MixtureKind{}}, options);
}
std::shared_ptr<nn::UnaryModule> sandwich(const Json& config, TensorOptions options) {
    return std::make_shared<nn::HybridDecoder>(
        config, nn::DecoderDesign{nn::NormKind::rms_from_one, nn::LoopEntry::joined, nn::LayerForm::sandwich, false, kSandwichMixers,
                                  nn::MixtureKind{.softmax = true, .correction = true, .gated = true, .weigh_results = true}, 1.702, true}, options);
}
std::shared_ptr<nn::UnaryModule> post_norm(const Json& config, TensorOptions options) {
    return std::make_shared<nn::HybridDecoder>(
        config, nn::DecoderDesign{nn::NormKind::rms, nn::LoopEntry::joined, nn::LayerForm::behind, false, kPostNormMixers,
                                  nn::MixtureKind{.gated = true, .weigh_results = true, .bias = true, .chosen_softmax = true}, 0.0, false, true, true}, options);
}

// Grouped-query decoder with its embedding and output layers, under the names of the reference's example model.
std::shared_ptr<nn::UnaryModule> transformer(const Json& c, TensorOptions options) {
    const bool tied = !c.has("tied") || c.at("tied").integer() != 0;
    return std::make_shared<nn::DecoderLanguageModel>(c.at("vocab").positive(), c.at("layers").positive(), c.at("width").positive(),
                                                      c.at("heads").positive(), c.at("kv_heads").positive(), c.at("ff").positive(),
                                                      c.at("context").positive(), tied, options);
}

struct Entry { const char* name; Factory make; };
constexpr Entry kRegistry[] = {
    {"Lozepel", sandwich},
    {"Ripitar", hybrid},
    {"Rizovik", post_norm},
    {"Sinezen", parallel},
    {"TransformerDecoder", transformer},
};

std::string read_text(const std::filesystem::path& path) {
    std::ifstream in(path, std::ios::binary);
    if (!in) throw std::runtime_error("cannot read " + path.string());
    std::ostringstream text;
    text << in.rdbuf();
    return text.str();
}

}  // namespace

std::vector<std::string> architectures() {
    std::vector<std::string> names;
    for (const auto& entry : kRegistry) names.emplace_back(entry.name);
    return names;
}

std::shared_ptr<nn::UnaryModule> create(const Json& config, TensorOptions options) {
    const std::string& name = config.at("architecture").text();
    for (const auto& entry : kRegistry)
        if (name == entry.name) return entry.make(config, options);
    throw std::invalid_argument("configuration: unknown architecture '" + name + "'");
}

std::shared_ptr<nn::UnaryModule> load(const std::filesystem::path& folder, DType dtype, Device device) {
    auto model = create(Json::parse(read_text(folder / "config.json")), {dtype, Device::cpu()});
    StateDict converted;
    for (auto& [name, tensor] : io::load_safetensors(folder / "model.safetensors")) {
        const bool floating = tensor.dtype() == DType::bf16 || tensor.dtype() == DType::f32 || tensor.dtype() == DType::f64;
        converted.emplace_back(name, floating ? tensor.astype(dtype) : tensor);
    }
    // buffers (position tables) are computed, not loaded
    for (const auto& [name, tensor] : model->state_dict()) {
        if (name.find("rotary.") == std::string::npos) continue;
        bool found = false;
        for (const auto& entry : converted) found = found || entry.first == name;
        if (!found) converted.emplace_back(name, tensor);
    }
    model->load_state_dict(converted);
    model->to(device);
    return model;
}

}  // namespace dl::models
