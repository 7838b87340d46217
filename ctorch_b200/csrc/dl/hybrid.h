// Configured decoders: a list of layers with their own mixers and feed-forwards, and a range of layers that may run several times in a
// row with the same weights.  Four designs are arranged from the pieces here (DecoderDesign; the registry holds them):
//   "Ripitar"  state-space (Mamba-2) and latent-attention layers, Dynamic Tanh norms, mixer and SwiGLU feed-forward one after the other;
//   "Sinezen"  chunked grouped-query attention beside a SwiGLU feed-forward or a mixture of experts that reads the same RMS norm;
//   "Lozepel"  a norm before and after every sublayer, three mixers (two kinds of grouped-query attention, and attention side by side with
//              lightning attention), clamped gated units or a mixture of gated experts, pair embedding, capped logits;
//   "Rizovik"  sublayers that read the stream itself, with norms behind them; attention over a window with pooled blocks before it, attention
//              over a window and the first tokens with mixed heads, the gated delta rule; a mixture of gated experts, tied embeddings, layers
//              that take over another one's weights.
//
// The pieces (norms, mixers, feed-forwards, looped range) are separate modules with their constants as parameters; HybridDecoder only
// arranges them.  Parameter names are the names of the weight files: "embed", "bigram", "head", "loop.step" or "loop.in",
// "final.norm{,.alpha,.b}", "l<i>.norm1{,.alpha,.b}", "l<i>.mix.*", "l<i>.mlp.*".  A layer with "weights_of": j in its configuration has no
// parameters of its own: it runs layer j's module once more, with a cache or state of its own.
#pragma once

#include "dl/dl.h"
#include "dl/json.h"
#include "dl/token_model.h"

#include <map>
#include <memory>
#include <optional>
#include <span>
#include <string>
#include <tuple>
#include <vector>

namespace dl::nn {

// (rms_from_one: the weight is stored as its distance from one)
enum class NormKind { dynamic_tanh, rms, rms_from_one };
// How a looped range is entered, before its first layer.
enum class LoopEntry {
    step,      // x + (embedding output, from the second pass on) + the pass's vector "loop.step"
    joined,    // "loop.in" [x; embedding output], in every pass
};
enum class LayerForm {
    sequential,   // mixer, then feed-forward, each behind its own norm
    parallel,     // mixer and feed-forward read one norm and are added together
    sandwich,     // sequential, with a norm behind each sublayer as well, before it is added
    behind,       // sequential, each sublayer reads the stream itself and has its norm behind it alone
};
enum class MixerKind { state_space, latent, attention, side_by_side, delta };
// "mask": runs of positions that begin at multiples of its size, or the last positions up to each one's own.
enum class AttentionMask { chunks, window };
enum class OutputGate { none, head, value };   // sigmoid(g) for every head, or for every value of a head
enum class Sink { none, zero, learned };   // a term of the softmax's denominator without a key
// What kinds of grouped-query attention differ in, beside the sizes and constants of the configuration.
struct AttentionKind {
    b200_head_norm norm = B200_HEAD_NORM_PROJECTION;
    bool rotate_pairs = false;     // entry 2i with entry 2i + 1; otherwise halves
    bool bias = false;             // on queries and keys
    bool keys_as_values = false;   // unrotated, the keys serve as values too
    OutputGate gate = OutputGate::none;
    Sink sink = Sink::none;
    AttentionMask mask = AttentionMask::chunks;
    bool head_weights = false;     // norm per head: with weights, the same for every head
    bool norm_values = false;      // every head's value over its root mean square
    bool talk = false;             // the heads' softmax weights are mixed by a matrix
};
struct MixtureKind {
    bool softmax = false;         // scores over all outputs together; otherwise sigmoid
    bool correction = false;      // a vector added to the scores for the choice alone
    bool gated = false;           // silu(gate x) * (up x); otherwise gelu(up x)
    bool weigh_results = false;   // the score multiplies the expert's result; otherwise its input
    bool bias = false;            // a vector added to the router's logits
    bool chosen_softmax = false;  // the largest logits are chosen, the scores are the softmax over them alone
};
// A layer type of a design's configurations and the mixer it stands for (`attention`: with that mixer, or the left one side by side).
struct MixerDesign {
    const char* type;
    MixerKind kind;
    AttentionKind attention = {};
};
// What the layers of a design have in common.
struct DecoderDesign {
    NormKind norm;
    LoopEntry loop;
    LayerForm form;
    bool scaled;                           // the configuration gives factors of the embedding and of the logits
    std::span<const MixerDesign> mixers;
    std::optional<MixtureKind> mixture;    // feed-forward kind "moe"
    double unit_slope = 0.0;               // dense feed-forward: clamped units with this slope, the limit from the configuration; 0: SwiGLU
    bool pairs = false;                    // rows of a table of token pairs are added to the embedding
    bool tied = false;                     // the logits come from the embedding table
    bool residual_factor = false;          // the configuration gives a factor of everything that is added to the stream
};

// Dynamic Tanh: tanh(alpha * x) * w + b; RMS norms: x / sqrt(mean(x^2) + eps) * w (or 1 + w), without alpha and bias.  The weight is the module's own
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

// Grouped-query attention, over all earlier positions, inside chunks of them, or over a window (0: none) and with it the first `keep`
// positions or means over blocks of `pool`; keys and values may differ in size.  With keys_from >= 0 the layer has no keys and values of its
// own and reads those of that layer.
struct GroupedAttentionConfig {
    Index heads, kv_heads, dim, vdim, chunk, rot_dims;
    double rot_base, scale;
    double softcap = 0.0;   // score <- softcap tanh(score / softcap); 0: as it is
    Index keys_from = -1;
    AttentionKind kind = {};
    Index window = 0, keep = 0, pool = 0;
    double rot_factor = 1.0;   // what the angles are divided by
};
class GroupedAttentionMixer : public Module {
public:
    GroupedAttentionMixer(Index width, const GroupedAttentionConfig& config, TensorOptions options);
    const GroupedAttentionConfig& config() const { return config_; }
    bool own_keys() const { return config_.keys_from < 0; }
    Index columns() const;   // rows of q, k, v and g together, as far as there are any
    Tensor *q, *k = nullptr, *v = nullptr, *q_norm = nullptr, *k_norm = nullptr, *q_bias = nullptr, *k_bias = nullptr, *sink = nullptr, *gate = nullptr, *out;
    Tensor* talk = nullptr;
private:
    GroupedAttentionConfig config_;
};

// Lightning attention: SiLU on queries, keys and values, S <- decay S + k v^T per head, o = S^T q; an RMS norm over all heads, a gate per value.
struct LightningConfig {
    Index heads, dim, vdim;
    std::vector<double> decay;   // [heads]
};
class LightningMixer : public Module {
public:
    LightningMixer(Index width, const LightningConfig& config, TensorOptions options);
    const LightningConfig& config() const { return config_; }
    Index inner() const { return config_.heads * config_.vdim; }
    Index channels() const { return inner() + 2 * config_.heads * config_.dim; }
    Tensor *q, *k, *v, *gate, *norm, *out;
private:
    LightningConfig config_;
};

// Gated delta rule: short convolutions with SiLU on queries, keys and values, unit queries and keys (kv_heads of them for `heads` values),
// S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; an RMS norm per head, times SiLU of a gate per value.
struct DeltaConfig { Index heads, kv_heads, dim, vdim, taps; };
class DeltaMixer : public Module {
public:
    DeltaMixer(Index width, const DeltaConfig& config, TensorOptions options);
    const DeltaConfig& config() const { return config_; }
    Index inner() const { return config_.heads * config_.vdim; }
    Index channels() const { return inner() + 2 * config_.kv_heads * config_.dim; }
    Tensor *q, *q_conv, *k, *k_conv, *v, *v_conv, *beta, *a_log, *norm, *rate, *dt_bias, *gate, *out;
private:
    DeltaConfig config_;
};

// Two mixers on one input; the results are added, each with its factor.
class SideBySideMixer : public Module {
public:
    SideBySideMixer(Index width, const GroupedAttentionConfig& left, const LightningConfig& right, double left_scale, double right_scale, TensorOptions options);
    std::shared_ptr<GroupedAttentionMixer> left;
    std::shared_ptr<LightningMixer> right;
    double left_scale, right_scale;
};

// Experts of which every token takes the `top` with the largest scores.  identity: further outputs of the router whose expert hands its
// input through.  shared_ff: units of an expert that runs for every token (0: none; gelu experts only).
struct MixtureConfig {
    Index experts, top, ff, shared_ff;
    Index identity = 0;
    MixtureKind kind = {};
    Index outputs() const { return experts + identity; }
};
class MixtureOfExperts : public Module {
public:
    MixtureOfExperts(Index width, const MixtureConfig& config, TensorOptions options);
    const MixtureConfig& config() const { return config_; }
    std::vector<Tensor*> gate, up, down;
    Tensor *router, *bias = nullptr, *correction = nullptr, *shared_up = nullptr, *shared_down = nullptr;
private:
    MixtureConfig config_;
};

class HybridLayer : public Module {
public:
    HybridLayer(Index width, const Json& spec, const DecoderDesign& design, TensorOptions options);
    RowNorm norm1, norm2;                           // before the sublayers; norm2 only with a feed-forward after the mixer
    RowNorm after1, after2;                         // behind the sublayers (sandwich, behind)
    std::shared_ptr<StateSpaceMixer> state_space;   // exactly one of the mixers, or attention and lightning
    std::shared_ptr<LatentAttentionMixer> latent;
    std::shared_ptr<GroupedAttentionMixer> attention;
    std::shared_ptr<DeltaMixer> delta;
    std::shared_ptr<LightningMixer> lightning;      // beside the attention, with their factors
    double attention_scale = 1.0, lightning_scale = 1.0;
    double unit_limit = 0.0;                        // clamped units of the dense feed-forward
    Tensor *gate = nullptr, *up = nullptr, *down = nullptr;   // dense feed-forward
    std::shared_ptr<MixtureOfExperts> mixture;
    bool has_mlp() const { return gate != nullptr; }
};

// One execution of a layer: looped layers run once per pass, each time with its own cache or state.
struct LayerRun {
    Index layer;         // number of its module in HybridDecoder::layers()
    Index pass;          // pass of the looped range, -1 outside
    bool begins_pass;    // first layer of a pass: the pass is entered before it (LoopEntry)
    Index keys_run;      // the run whose keys and values it reads (attention: its own, or one before it)
};

// What the decoder keeps per sequence: slots of equal capacity, each with its length; per layer run a paged latent cache, a
// convolution ring and a recurrent state, or the keys and values of one chunk, or of one window with what stands before it (of the whole
// sequence without either); and the last token, where the embedding reads it.  A slot is given back by release(); its next sequence starts at position 0, where the
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
        Tensor key, value;       // [slots, kv_heads, entries, dim | vdim]; none where another run's are read
        Tensor pool;             // [slots, kv_heads, dim + vdim]: sums of the block that is being pooled
        Index entries = 0;
        Index window = 0, keep = 0, pools = 0;   // as far as the capacity lets a position see less than everything
    };
    const Run& run(std::size_t i) const { return runs_[i]; }
    std::int32_t* lengths() const { return static_cast<std::int32_t*>(lengths_.mutable_data()); }
    std::int32_t* last_tokens() const { return static_cast<std::int32_t*>(last_.mutable_data()); }
    void commit(Index slot, Index count) { lengths_host_[static_cast<std::size_t>(slot)] += count; }
    struct Rotary { Tensor cosine, sine; };
    const Rotary& rotary(Index dims, double base, double factor = 1.0) const { return tables_.at({dims, base, factor}); }

private:
    void set_length(Index slot, std::int32_t length);
    Index capacity_;
    int device_;
    std::uint64_t id_;
    Tensor lengths_, last_;    // int32 payload [slots]
    std::vector<Index> lengths_host_;
    std::vector<Run> runs_;
    std::map<std::tuple<Index, double, double>, Rotary> tables_;
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
    double logit_softcap() const { return logit_softcap_; }   // 0: none
    double residual_factor() const { return residual_factor_; }
    // Table of token pairs (NULL: none), [buckets + 1, width]; the pair's row is (previous * mul_prev + token * mul_cur) mod buckets.
    const Tensor* pairs() const { return pairs_; }
    struct PairHash { Index buckets, mul_prev, mul_cur; };
    const PairHash& pair_hash() const { return pair_hash_; }
    // The layers with weights of their own, in the order of the configuration.
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
    double eps_, embedding_scale_, logit_scale_, logit_softcap_ = 0.0, residual_factor_ = 1.0;
    PairHash pair_hash_{};
    Tensor *embed_, *head_, *pairs_ = nullptr, *loop_step_ = nullptr, *loop_in_ = nullptr;
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
