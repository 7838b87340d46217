// Configured decoders: a list of layers with their own mixers and feed-forwards, and a range of layers that may run several times in a
// row with the same weights.  Two designs are arranged from the pieces here (DecoderDesign):
//   "Ripitar"  state-space (Mamba-2) and latent-attention layers, Dynamic Tanh norms, mixer and SwiGLU feed-forward one after the other;
//   "Sinezen"  chunked grouped-query attention beside a SwiGLU feed-forward or a mixture of experts that reads the same RMS norm.
//
// The pieces (norms, mixers, feed-forwards, looped range) are separate modules with their constants as parameters; HybridDecoder only
// arranges them.  Parameter names are the names of the weight files: "embed", "head", "loop.step" or "loop.in",
// "final.norm{,.alpha,.b}", "l<i>.norm1{,.alpha,.b}", "l<i>.mix.*", "l<i>.mlp.*".
#pragma once

#include "dl/dl.h"
#include "dl/json.h"
#include "dl/token_model.h"

#include <map>
#include <memory>
#include <span>
#include <string>
#include <vector>

namespace dl::nn {

enum class NormKind { dynamic_tanh, rms };
// How a looped range is entered, before its first layer.
enum class LoopEntry {
    step,      // x + (embedding output, from the second pass on) + the pass's vector "loop.step"
    joined,    // "loop.in" [x; embedding output], in every pass
};
// What the layers of a design have in common.
struct DecoderDesign {
    NormKind norm;
    LoopEntry loop;
    bool parallel;   // mixer and feed-forward read one norm and are added together
    bool scaled;     // the configuration gives factors of the embedding and of the logits
};

// Dynamic Tanh: tanh(alpha * x) * w + b; RMS norm: x / sqrt(mean(x^2) + eps) * w, without alpha and bias.  The weight is the module's own
// name, alpha and bias beside it, so the names live in the parent.
struct RowNorm {
    Tensor *weight = nullptr, *alpha = nullptr, *bias = nullptr;
    bool rms() const { return alpha == nullptr; }
};

struct StateSpaceConfig { Index heads, vdim, state, groups, taps, norm_groups; };
struct LatentAttentionConfig {
    Index heads, dim, rot_dim, vdim, kv_rank, q_rank, rot_dims;
    double rot_base, scale;
};

class StateSpaceMixer : public Module {
public:
    StateSpaceMixer(Index width, const StateSpaceConfig& config, TensorOptions options);
    const StateSpaceConfig& config() const { return config_; }
    Index inner() const { return config_.heads * config_.vdim; }
    Index channels() const { return inner() + 2 * config_.groups * config_.state; }
    Tensor *in, *conv, *conv_bias, *dt_bias, *a_log, *d, *norm, *out;
private:
    StateSpaceConfig config_;
};

class LatentAttentionMixer : public Module {
public:
    LatentAttentionMixer(Index width, const LatentAttentionConfig& config, TensorOptions options);
    const LatentAttentionConfig& config() const { return config_; }
    Tensor *dq, *dq_norm, *uq, *dkv, *dkv_norm, *uk, *uv, *gate, *out;
private:
    LatentAttentionConfig config_;
};

// Grouped-query attention inside chunks of positions (0: none), RMS norms over all query heads and over all key heads, rotation of
// halves, one output gate per head; keys and values may differ in size.
struct ChunkedAttentionConfig {
    Index heads, kv_heads, dim, vdim, chunk, rot_dims;
    double rot_base, scale;
};
class ChunkedAttentionMixer : public Module {
public:
    ChunkedAttentionMixer(Index width, const ChunkedAttentionConfig& config, TensorOptions options);
    const ChunkedAttentionConfig& config() const { return config_; }
    Index columns() const;   // rows of q, k, v and g together
    Tensor *q, *k, *v, *q_norm, *k_norm, *gate, *out;
private:
    ChunkedAttentionConfig config_;
};

// Experts down gelu(up x) of which every token takes the `top` with the largest sigmoid scores; the score multiplies the expert's
// input.  shared_ff: units of an expert of the same form that runs for every token (0: none).
struct MixtureConfig { Index experts, top, ff, shared_ff; };
class MixtureOfExperts : public Module {
public:
    MixtureOfExperts(Index width, const MixtureConfig& config, TensorOptions options);
    const MixtureConfig& config() const { return config_; }
    std::vector<Tensor*> up, down;
    Tensor *router, *shared_up = nullptr, *shared_down = nullptr;
private:
    MixtureConfig config_;
};

class HybridLayer : public Module {
public:
    HybridLayer(Index width, const Json& spec, const DecoderDesign& design, TensorOptions options);
    RowNorm norm1, norm2;                           // norm2 only with a feed-forward after the mixer
    std::shared_ptr<StateSpaceMixer> state_space;   // exactly one of the mixers
    std::shared_ptr<LatentAttentionMixer> latent;
    std::shared_ptr<ChunkedAttentionMixer> chunked;
    Tensor *gate = nullptr, *up = nullptr, *down = nullptr;   // dense feed-forward
    std::shared_ptr<MixtureOfExperts> mixture;
    bool has_mlp() const { return gate != nullptr; }
};

// One execution of a layer: looped layers run once per pass, each time with its own cache or state.
struct LayerRun {
    Index layer;
    Index pass;          // pass of the looped range, -1 outside
    bool begins_pass;    // first layer of a pass: the pass is entered before it (LoopEntry)
};

// What the decoder keeps per sequence: slots of equal capacity, each with its length; per layer run a paged latent cache, a
// convolution ring and a recurrent state, or the keys and values of one chunk.  A slot is given back by release(); its next sequence starts at position 0, where the
// kernels read nothing old.
class HybridDecoder;
class HybridCache {
public:
    HybridCache(const HybridDecoder& model, Index slots, Index capacity);
    ~HybridCache();
    HybridCache(const HybridCache&) = delete;
    HybridCache& operator=(const HybridCache&) = delete;
    Index slots() const { return static_cast<Index>(lengths_host_.size()); }
    Index capacity() const { return capacity_; }
    Index length(Index slot) const;
    Index longest() const;
    void release(Index slot);
    void clear();
    int device() const { return device_; }
    std::uint64_t id() const { return id_; }

    // used by the plan
    struct Run {
        b200_kv_cache* latent = nullptr;
        Tensor conv, state;      // [slots, taps, channels], [slots, heads, state, vdim]
        Tensor key, value;       // [slots, kv_heads, entries, dim | vdim]
        Index entries = 0;
    };
    const Run& run(std::size_t i) const { return runs_[i]; }
    std::int32_t* lengths() const { return static_cast<std::int32_t*>(lengths_.mutable_data()); }
    void commit(Index slot, Index count) { lengths_host_[static_cast<std::size_t>(slot)] += count; }
    struct Rotary { Tensor cosine, sine; };
    const Rotary& rotary(Index dims, double base) const { return tables_.at({dims, base}); }

private:
    void set_length(Index slot, std::int32_t length);
    Index capacity_;
    int device_;
    std::uint64_t id_;
    Tensor lengths_;    // int32 payload [slots]
    std::vector<Index> lengths_host_;
    std::vector<Run> runs_;
    std::map<std::pair<Index, double>, Rotary> tables_;
};

// One sequence's share of a pass: its next tokens, and which of them (indices into tokens) the caller wants logits of.
struct PassEntry {
    Index slot;
    std::span<const Index> tokens;
    std::span<const Index> want;
};

class HybridPlan;

class HybridDecoder : public UnaryModule {
public:
    HybridDecoder(const Json& config, const DecoderDesign& design, TensorOptions options = {});
    ~HybridDecoder() override;
    // ids [batch, length] -> logits [batch, length, vocabulary] f32, without a cache that outlives the call
    Tensor forward(const Tensor& ids) override;
    // Runs the entries as one packed pass from what earlier passes left in their slots; logits of the wanted tokens to the host
    // buffer [wanted, vocabulary] in the order of entries and wants.  `trail` (tests) receives the residual stream [rows, width]
    // after every layer run.
    void pass(HybridCache& cache, std::span<const PassEntry> entries, float* logits, std::vector<float>* trail = nullptr);

    Index width() const { return width_; }
    Index vocabulary() const { return vocab_; }
    DType dtype() const { return dtype_; }
    double eps() const { return eps_; }
    double embedding_scale() const { return embedding_scale_; }
    double logit_scale() const { return logit_scale_; }
    const std::vector<std::shared_ptr<HybridLayer>>& layers() const { return layers_; }
    const std::vector<LayerRun>& runs() const { return runs_; }
    const Tensor& embed() const { return *embed_; }
    const Tensor& head() const { return *head_; }
    const DecoderDesign& design() const { return design_; }
    const Tensor* loop_step() const { return loop_step_; }
    const Tensor* loop_in() const { return loop_in_; }
    const RowNorm& final_norm() const { return final_norm_; }
    // As TransformerDecoder::set_activation_dtype: bf16 drops the lo plane of the projections' inputs in passes over more than 16 rows.
    void set_activation_dtype(DType dtype);
    DType activation_dtype() const { return activation_dtype_; }
    HybridPlan& plan();

private:
    Index width_, vocab_;
    DType dtype_, activation_dtype_ = DType::f32;
    DecoderDesign design_;
    double eps_, embedding_scale_, logit_scale_;
    Tensor *embed_, *head_, *loop_step_ = nullptr, *loop_in_ = nullptr;
    RowNorm final_norm_;
    std::vector<std::shared_ptr<HybridLayer>> layers_;
    std::vector<LayerRun> runs_;
    std::unique_ptr<HybridPlan> plan_;
};

// A configured decoder behind the generation loop: sequence b of the batch lives in slot b.
std::unique_ptr<TokenModel> make_token_model(std::shared_ptr<HybridDecoder> model, std::shared_ptr<HybridCache> cache);

}  // namespace dl::nn

namespace dl::models {

// Registry of model designs by the "architecture" of their configuration.
std::vector<std::string> architectures();
std::shared_ptr<nn::UnaryModule> create(const Json& config, TensorOptions options);
// config.json and model.safetensors of a folder, weights converted to `dtype` (bf16 or f32), on `device`.
std::shared_ptr<nn::UnaryModule> load(const std::filesystem::path& folder, DType dtype, Device device);

}  // namespace dl::models
