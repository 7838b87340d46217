// Modules, cache, execution plan and generation of the configured decoders (see hybrid.h, hybrid_plan.h; parallel layers: parallel.cpp,
// layers with norms behind the sublayers: sandwich.cpp, delta.cpp).
#include "dl/hybrid_plan.h"

#include <algorithm>
#include <atomic>
#include <cmath>
#include <stdexcept>

namespace dl::nn {

namespace {
constexpr Index kPassRows = 8192;          // rows of one pass over the layers; longer passes are cut
constexpr Index kPageSize = 64;
}  // namespace

// ---- modules ------------------------------------------------------------------------------------------------
StateSpaceMixer::StateSpaceMixer(Index width, const StateSpaceConfig& c, TensorOptions options) : config_(c) {
    if (c.heads % c.groups) throw std::invalid_argument("state-space mixer: heads must be a multiple of groups");
    if (inner() % c.norm_groups) throw std::invalid_argument("state-space mixer: heads * vdim must be a multiple of norm_groups");
    if (c.state > B200_SSM_MAX_STATE) throw std::invalid_argument("state-space mixer: the state size exceeds " + std::to_string(B200_SSM_MAX_STATE));
    in = &register_parameter("in", host_zeros({inner() + channels() + c.heads, width}, options));
    conv = &register_parameter("conv", host_zeros({channels(), c.taps}, options));
    conv_bias = &register_parameter("conv.b", host_zeros({channels()}, options));
    dt_bias = &register_parameter("dt_bias", host_zeros({c.heads}, options));
    a_log = &register_parameter("A_log", host_zeros({c.heads}, options));
    d = &register_parameter("D", host_zeros({c.heads}, options));
    norm = &register_parameter("norm", ones({inner()}, options));
    out = &register_parameter("o", host_zeros({width, inner()}, options));
}

LatentAttentionMixer::LatentAttentionMixer(Index width, const LatentAttentionConfig& c, TensorOptions options) : config_(c) {
    if (c.rot_dims % 2 || c.rot_dims > c.rot_dim) throw std::invalid_argument("latent attention: rotated dimensions must be even and at most rot_dim");
    dq = &register_parameter("dq", host_zeros({c.q_rank, width}, options));
    dq_norm = &register_parameter("dq.norm", ones({c.q_rank}, options));
    uq = &register_parameter("uq", host_zeros({c.heads * (c.dim + c.rot_dim), c.q_rank}, options));
    dkv = &register_parameter("dkv", host_zeros({c.kv_rank + c.rot_dim, width}, options));
    dkv_norm = &register_parameter("dkv.norm", ones({c.kv_rank}, options));
    uk = &register_parameter("uk", host_zeros({c.heads * c.dim, c.kv_rank}, options));
    uv = &register_parameter("uv", host_zeros({c.heads * c.vdim, c.kv_rank}, options));
    gate = &register_parameter("g", host_zeros({c.heads * c.vdim, width}, options));
    out = &register_parameter("o", host_zeros({width, c.heads * c.vdim}, options));
}

namespace {
GroupedAttentionConfig attention_config(const Json& m, const AttentionKind& kind) {
    GroupedAttentionConfig c{m.at("heads").positive(), m.at("kv_heads").positive(), m.at("dim").positive(), m.at("vdim").positive(), 0, 0, 1.0,
                             m.at("scale").number()};
    c.kind = kind;
    if (m.has("mask")) {
        const Json& mask = m.at("mask");
        (kind.mask == AttentionMask::chunks ? c.chunk : c.window) = mask.at("size").positive();
        if (kind.mask == AttentionMask::window) {
            if (mask.has("keep_first")) c.keep = mask.at("keep_first").integer();
            if (mask.has("pool")) c.pool = mask.at("pool").positive();
            if (c.keep < 0) throw std::invalid_argument("configuration: 'keep_first' must not be negative");
        }
    }
    if (m.has("rot")) {
        const Json& rot = m.at("rot");
        c.rot_dims = rot.at("dims").positive();
        c.rot_base = rot.at("base").number();
        if (rot.has("scaling")) c.rot_factor = rot.at("scaling").at("factor").number();
        if (!(c.rot_factor > 0.0)) throw std::invalid_argument("configuration: the scaling 'factor' must be positive");
    }
    if (m.has("softcap")) {
        c.softcap = m.at("softcap").number();
        if (!(c.softcap > 0.0)) throw std::invalid_argument("configuration: 'softcap' must be positive");
    }
    if (m.has("kv_from")) {
        c.keys_from = m.at("kv_from").integer();
        if (c.keys_from < 0) throw std::invalid_argument("configuration: 'kv_from' must be the number of a layer");
    }
    return c;
}
LightningConfig lightning_config(const Json& m) {
    LightningConfig c{m.at("heads").positive(), m.at("dim").positive(), m.at("vdim").positive(), {}};
    for (const Json& d : m.at("decay").items()) c.decay.push_back(d.number());
    return c;
}
}  // namespace

HybridLayer::HybridLayer(Index width, const Json& spec, const DecoderDesign& design, TensorOptions options) {
    auto norm = [&](const std::string& name) {
        RowNorm n;
        n.weight = &register_parameter(name, ones({width}, options));
        if (design.norm != NormKind::dynamic_tanh) return n;
        n.bias = &register_parameter(name + ".b", host_zeros({width}, options));
        n.alpha = &register_parameter(name + ".alpha", ones({}, options));
        return n;
    };
    const bool sandwich = design.form == LayerForm::sandwich, behind = design.form == LayerForm::behind;
    (behind ? after1 : norm1) = norm("norm1");
    if (sandwich) after1 = norm("norm1b");
    const std::string& type = spec.at("type").text();
    const auto mixer = std::find_if(design.mixers.begin(), design.mixers.end(), [&](const MixerDesign& d) { return type == d.type; });
    if (mixer == design.mixers.end()) throw std::invalid_argument("configuration: unknown layer type '" + type + "' of this architecture");
    const Json& m = spec.at("mixer");
    switch (mixer->kind) {
    case MixerKind::state_space: {
        const StateSpaceConfig c{m.at("heads").positive(), m.at("vdim").positive(), m.at("state").positive(), m.at("groups").positive(),
                                 m.at("conv").positive(), m.at("norm_groups").positive()};
        state_space = add_module<StateSpaceMixer>("mix", width, c, options);
        break;
    }
    case MixerKind::latent: {
        const Json& rot = m.at("rot");
        const LatentAttentionConfig c{m.at("heads").positive(), m.at("dim").positive(), m.at("rot_dim").positive(), m.at("vdim").positive(),
                                      m.at("kv_rank").positive(), m.at("q_rank").positive(), rot.at("dims").positive(), rot.at("base").number(),
                                      m.at("scale").number()};
        latent = add_module<LatentAttentionMixer>("mix", width, c, options);
        break;
    }
    case MixerKind::attention:
        attention = add_module<GroupedAttentionMixer>("mix", width, attention_config(m, mixer->attention), options);
        break;
    case MixerKind::side_by_side: {
        const auto pair = add_module<SideBySideMixer>("mix", width, attention_config(m.at("left"), mixer->attention), lightning_config(m.at("right")),
                                                      m.at("left_scale").number(), m.at("right_scale").number(), options);
        attention = pair->left;
        lightning = pair->right;
        attention_scale = pair->left_scale;
        lightning_scale = pair->right_scale;
        break;
    }
    case MixerKind::delta:
        delta = add_module<DeltaMixer>("mix", width, DeltaConfig{m.at("heads").positive(), m.at("kv_heads").positive(), m.at("dim").positive(),
                                                                 m.at("vdim").positive(), m.at("conv").positive()}, options);
        break;
    }
    if (!spec.has("mlp")) return;
    const Json& mlp = spec.at("mlp");
    const std::string& kind = mlp.at("kind").text();
    if (design.form != LayerForm::parallel) (behind ? after2 : norm2) = norm("norm2");
    if (sandwich) after2 = norm("norm2b");
    if (design.mixture && kind == "moe") {
        const Json& router = mlp.at("router");
        MixtureConfig c{router.at("experts").positive(), router.at("top").positive(), mlp.at("expert").at("ff").positive(),
                        mlp.has("shared") ? mlp.at("shared").at("ff").positive() : 0};
        c.kind = *design.mixture;
        if (router.has("identity")) c.identity = router.at("identity").integer();
        mixture = add_module<MixtureOfExperts>("mlp", width, c, options);
        return;
    }
    if (kind != "dense") throw std::invalid_argument("configuration: unknown feed-forward kind '" + kind + "'");
    const Index ff = mlp.at("ff").positive();
    if (design.unit_slope > 0.0) {
        unit_limit = mlp.at("limit").number();
        if (!(unit_limit > 0.0)) throw std::invalid_argument("configuration: 'limit' must be positive");
    }
    gate = &register_parameter("mlp.gate", host_zeros({ff, width}, options));
    up = &register_parameter("mlp.up", host_zeros({ff, width}, options));
    down = &register_parameter("mlp.down", host_zeros({width, ff}, options));
}

void HybridDecoder::set_activation_dtype(DType dtype) {
    if (dtype != DType::f32 && dtype != DType::bf16) throw std::invalid_argument("activation dtype must be f32 or bf16");
    if (dtype == DType::bf16 && dtype_ != DType::bf16) throw std::invalid_argument("bf16 activations need a bf16 decoder");
    activation_dtype_ = dtype;
}

// ---- cache --------------------------------------------------------------------------------------------------
namespace {
std::atomic<std::uint64_t> hybrid_cache_ids{1};

// cos / sin of position * base^(-2i/dims) / factor, computed in f64 on the host and rounded once.
HybridCache::Rotary rotary_table(Index dims, double base, double factor, Index positions, Device device) {
    if (base <= 0) throw std::invalid_argument("rotary base must be positive");
    const Index half = dims / 2;
    Tensor cosine = empty({positions, half}, {DType::f32, Device::cpu()}), sine = empty({positions, half}, {DType::f32, Device::cpu()});
    for (Index i = 0; i < half; ++i) {
        const double frequency = std::pow(base, -2.0 * static_cast<double>(i) / static_cast<double>(dims)) / factor;
        for (Index p = 0; p < positions; ++p) {
            f32(cosine)[p * half + i] = static_cast<float>(std::cos(static_cast<double>(p) * frequency));
            f32(sine)[p * half + i] = static_cast<float>(std::sin(static_cast<double>(p) * frequency));
        }
    }
    return {cosine.to(device), sine.to(device)};
}
}  // namespace

HybridCache::HybridCache(const HybridDecoder& model, Index slots, Index capacity)
    : capacity_(capacity), device_(model.embed().device().index), id_(hybrid_cache_ids.fetch_add(1)) {
    if (slots <= 0 || capacity <= 0) throw std::invalid_argument("a cache needs at least one slot and a positive capacity");
    if (model.embed().device().type != DeviceType::cuda)
        throw std::invalid_argument("HybridDecoder: tensors must live on a CUDA device (this library has no CPU compute path)");
    runtime::set_device(device_);
    const Device where = Device::cuda(device_);
    lengths_host_.assign(static_cast<std::size_t>(slots), 0);
    lengths_ = zeros({slots}, {DType::f32, where});   // all-zero bits: int32 zeros
    if (model.pairs()) last_ = zeros({slots}, {DType::f32, where});
    auto rotary = [&](Index dims, double base, double factor = 1.0) {
        auto& table = tables_[{dims, base, factor}];
        if (!table.cosine.defined()) table = rotary_table(dims, base, factor, capacity, where);
    };
    try {
        for (const auto& r : model.runs()) {
            const HybridLayer& layer = *model.layers()[static_cast<std::size_t>(r.layer)];
            runs_.emplace_back();
            Run& run = runs_.back();
            if (layer.latent) {
                const auto& c = layer.latent->config();
                runtime::check(b200_latent_cache_create(device_, code_of(model.dtype()), static_cast<int32_t>(slots),
                                                        static_cast<int32_t>(c.kv_rank + c.rot_dim), static_cast<int32_t>(capacity), kPageSize,
                                                        lengths(), &run.latent), "latent cache allocation");
                rotary(c.rot_dims, c.rot_base);
            } else if (layer.attention) {
                const auto& c = layer.attention->config();
                run.entries = c.chunk > 0 ? std::min(c.chunk, capacity) : capacity;
                if (c.window > 0 && c.window < capacity && c.keep + c.window < capacity) {   // (otherwise every position sees all before it)
                    run.window = c.window;
                    run.keep = c.keep;
                    run.pools = c.pool;
                    run.entries = c.keep + c.window + (c.pool > 0 ? capacity / c.pool : 0);
                    if (c.pool > 0) run.pool = empty({slots, c.kv_heads, c.dim + c.vdim}, {DType::f32, where});
                }
                if (layer.attention->own_keys()) {
                    run.key = empty({slots, c.kv_heads, run.entries, c.dim}, {model.dtype(), where});
                    run.value = empty({slots, c.kv_heads, run.entries, c.vdim}, {model.dtype(), where});
                }
                if (c.rot_dims > 0) rotary(c.rot_dims, c.rot_base, c.rot_factor);
                if (layer.lightning) {
                    const auto& r = layer.lightning->config();
                    run.state = empty({slots, r.heads, r.dim, r.vdim}, {DType::f32, where});
                }
            } else if (layer.delta) {
                const auto& c = layer.delta->config();
                run.conv = empty({slots, c.taps, layer.delta->channels()}, {DType::f32, where});
                run.state = empty({slots, c.heads, c.dim, c.vdim}, {DType::f32, where});
            } else {
                const auto& c = layer.state_space->config();
                run.conv = empty({slots, c.taps, layer.state_space->channels()}, {DType::f32, where});
                run.state = empty({slots, c.heads, c.state, c.vdim}, {DType::f32, where});
            }
        }
    } catch (...) {
        for (auto& run : runs_) b200_kv_cache_release(run.latent);
        throw;
    }
}
HybridCache::~HybridCache() {
    try { synchronize(Device::cuda(device_)); } catch (...) {}
    for (auto& run : runs_) b200_kv_cache_release(run.latent);
}
Index HybridCache::length(Index slot) const {
    if (slot < 0 || slot >= slots()) throw std::out_of_range("cache slot out of range");
    return lengths_host_[static_cast<std::size_t>(slot)];
}
Index HybridCache::longest() const { return *std::max_element(lengths_host_.begin(), lengths_host_.end()); }
void HybridCache::set_length(Index slot, std::int32_t length) {
    lengths_host_[static_cast<std::size_t>(slot)] = length;
    runtime::copy_bytes(lengths() + slot, Device::cuda(device_), &length, Device::cpu(), sizeof length);
}
void HybridCache::release(Index slot) {
    length(slot);
    set_length(slot, 0);
}
void HybridCache::clear() { for (Index s = 0; s < slots(); ++s) set_length(s, 0); }

// ---- decoder ------------------------------------------------------------------------------------------------
HybridDecoder::HybridDecoder(const Json& config, const DecoderDesign& design, TensorOptions options)
    : width_(config.at("width").positive()), vocab_(config.at("vocab").positive()), dtype_(options.dtype), design_(design),
      eps_(config.at("norm").at("eps").number()), embedding_scale_(design.scaled ? config.at("embedding").at("scale").number() : 1.0),
      logit_scale_(design.scaled ? config.at("logit_scale").number() : 1.0) {
    if (dtype_ != DType::f32 && dtype_ != DType::bf16) throw std::invalid_argument("the B200 decoder path stores weights in f32 or bf16");
    if (config.has("logit_softcap")) {
        logit_softcap_ = config.at("logit_softcap").number();
        if (!(logit_softcap_ > 0.0)) throw std::invalid_argument("configuration: 'logit_softcap' must be positive");
    }
    if (design_.residual_factor) residual_factor_ = config.at("residual_mult").number();
    embed_ = &register_parameter("embed", host_zeros({vocab_, width_}, options));
    if (design_.pairs) {
        const Json& pair = config.at("embedding").at("bigram");
        pair_hash_ = {pair.at("buckets").positive(), pair.at("mul_prev").integer(), pair.at("mul_cur").integer()};
        pairs_ = &register_parameter("bigram", host_zeros({pair_hash_.buckets + 1, width_}, options));
    }
    if ((design_.form == LayerForm::sandwich || design_.form == LayerForm::behind) && config.has("loop"))
        throw std::invalid_argument("configuration: looped layers are not combined with norms behind the sublayers");
    const auto& specs = config.at("layers").items();
    const auto count = static_cast<Index>(specs.size());
    if (count == 0) throw std::invalid_argument("decoder requires at least one layer");
    std::vector<Index> module_of(static_cast<std::size_t>(count), -1);   // the module that a layer of the configuration runs
    for (Index i = 0; i < count; ++i) {
        const Json& spec = specs[static_cast<std::size_t>(i)];
        if (spec.has("weights_of")) continue;
        module_of[static_cast<std::size_t>(i)] = static_cast<Index>(layers_.size());
        layers_.push_back(add_module<HybridLayer>("l" + std::to_string(i), width_, spec, design_, options));
    }
    for (Index i = 0; i < count; ++i) {
        Index from = i;
        for (Index hops = 0; specs[static_cast<std::size_t>(from)].has("weights_of"); ++hops) {
            from = specs[static_cast<std::size_t>(from)].at("weights_of").integer();
            if (from < 0 || from >= count || hops >= count) throw std::invalid_argument("configuration: 'weights_of' must name a layer with weights");
        }
        if (specs[static_cast<std::size_t>(i)].at("type").text() != specs[static_cast<std::size_t>(from)].at("type").text())
            throw std::invalid_argument("configuration: 'weights_of' must name a layer of the same type");
        module_of[static_cast<std::size_t>(i)] = module_of[static_cast<std::size_t>(from)];
    }
    Index start = 0, stop = 0, times = 0;
    if (config.has("loop")) {
        start = config.at("loop").at("start").integer();
        stop = config.at("loop").at("stop").integer();
        times = config.at("loop").at("times").positive();
        if (start < 0 || stop < start || stop > count) throw std::invalid_argument("configuration: 'loop' must name a range of layers");
        if ((design_.loop == LoopEntry::joined) != (design_.norm != NormKind::dynamic_tanh))
            throw std::invalid_argument("this entry of a looped range is not combined with these norms");
        if (design_.loop == LoopEntry::step) loop_step_ = &register_parameter("loop.step", host_zeros({times, width_}, options));
        else loop_in_ = &register_parameter("loop.in", host_zeros({width_, 2 * width_}, options));
    }
    auto add_run = [&](Index number, Index pass, bool begins) {
        const auto own = static_cast<Index>(runs_.size());
        const Index layer = module_of[static_cast<std::size_t>(number)];
        const auto& mixer = layers_[static_cast<std::size_t>(layer)]->attention;
        if (!mixer || mixer->own_keys()) return runs_.push_back({layer, pass, begins, own});
        // the latest run of the layer it names
        const auto& c = mixer->config();
        const Index wanted = c.keys_from < count ? module_of[static_cast<std::size_t>(c.keys_from)] : -1;
        Index from = own - 1;
        while (from >= 0 && runs_[static_cast<std::size_t>(from)].layer != wanted) --from;
        const auto& source = from >= 0 ? layers_[static_cast<std::size_t>(wanted)]->attention : nullptr;
        if (!source || !source->own_keys() || source->config().kv_heads != c.kv_heads || source->config().dim != c.dim || source->config().vdim != c.vdim
            || source->config().chunk != c.chunk)
            throw std::invalid_argument("configuration: 'kv_from' must name an earlier attention layer with keys of its own and of the same sizes");
        runs_.push_back({layer, pass, begins, from});
    };
    for (Index i = 0; i < start; ++i) add_run(i, -1, false);
    for (Index t = 0; t < times; ++t)
        for (Index i = start; i < stop; ++i) add_run(i, t, i == start);
    for (Index i = stop; i < count; ++i) add_run(i, -1, false);
    final_norm_.weight = &register_parameter("final.norm", ones({width_}, options));
    if (design_.norm == NormKind::dynamic_tanh) {
        final_norm_.bias = &register_parameter("final.norm.b", host_zeros({width_}, options));
        final_norm_.alpha = &register_parameter("final.norm.alpha", ones({}, options));
    }
    head_ = design_.tied ? embed_ : &register_parameter("head", host_zeros({vocab_, width_}, options));
}

HybridDecoder::~HybridDecoder() = default;
HybridPlan& HybridDecoder::plan() {
    if (!plan_) plan_ = std::make_unique<HybridPlan>(*this);
    return *plan_;
}

Tensor to_f32(const Tensor& t) { return t.to(Device::cpu()).astype(DType::f32).to(t.device()); }

namespace {
// [heads * dim, rank] -> per head [rank, dim]
Tensor transpose_heads(const Tensor& w, Index heads, Index dim, Index rank) {
    const Tensor host = w.to(Device::cpu());
    Tensor result = empty({heads * rank, dim}, {w.dtype(), Device::cpu()});
    auto move = [&](auto* to, const auto* from) {
        for (Index h = 0; h < heads; ++h)
            for (Index d = 0; d < dim; ++d)
                for (Index r = 0; r < rank; ++r) to[(h * rank + r) * dim + d] = from[(h * dim + d) * rank + r];
    };
    if (w.dtype() == DType::bf16) move(static_cast<std::uint16_t*>(result.mutable_data()), host.data<std::uint16_t>());
    else move(static_cast<float*>(result.mutable_data()), host.data<float>());
    return result.to(w.device());
}
}  // namespace

HybridPlan::Norm HybridPlan::pack_norm(const RowNorm& n, double scale) const {
    Norm packed;
    auto scaled = [&](const Tensor& t) {
        Tensor host = t.to(Device::cpu()).astype(DType::f32).clone();
        const double from = &t == n.weight && owner_.design().norm == NormKind::rms_from_one ? 1.0 : 0.0;
        for (Index i = 0; i < host.numel(); ++i) f32(host)[i] = static_cast<float>((static_cast<double>(f32(host)[i]) + from) * scale);
        return host.to(t.device());
    };
    packed.weight = scaled(*n.weight);
    packed.rms = n.rms();
    if (packed.rms) return packed;
    packed.bias = scaled(*n.bias);
    packed.alpha = n.alpha->to(Device::cpu()).astype(DType::f32).data<float>()[0];
    return packed;
}

void HybridPlan::refresh() {
    const auto version = owner_.version();
    if (version == packed_version_ && !layers_.empty()) return;
    if (owner_.embed().device().type != DeviceType::cuda)
        throw std::invalid_argument("HybridDecoder: tensors must live on a CUDA device (this library has no CPU compute path)");
    runtime::set_device(device());
    synchronize(Device::cuda(device()));
    layers_.clear();
    for (const auto& module : owner_.layers()) {
        Layer l{};
        if (module->norm1.weight) l.norm1 = pack_norm(module->norm1);
        if (module->after1.weight || module->attention) {
            if (module->after1.weight) pack_sandwich(*module, l);
            else pack_parallel(*module, l);
            layers_.push_back(std::move(l));
            continue;
        }
        if (module->state_space) {
            const StateSpaceMixer& m = *module->state_space;
            l.in = m.in->raw_data(); l.out = m.out->raw_data();
            l.wide_out = m.inner() + m.channels() + m.config().heads;
            l.inner = m.inner();
            l.conv = to_f32(*m.conv); l.conv_bias = to_f32(*m.conv_bias); l.dt_bias = to_f32(*m.dt_bias);
            l.a_log = to_f32(*m.a_log); l.d = to_f32(*m.d); l.gated_norm = to_f32(*m.norm);
        } else {
            const LatentAttentionMixer& m = *module->latent;
            const auto& c = m.config();
            const Tensor parts[3] = {*m.dq, *m.dkv, *m.gate};
            l.wide = concat_rows(parts);
            l.in = l.wide.raw_data(); l.out = m.out->raw_data();
            l.wide_out = l.wide.size(0);
            l.inner = c.heads * c.vdim;
            l.uq = m.uq->raw_data(); l.w_value = m.uv->raw_data();
            l.w_key = transpose_heads(*m.uk, c.heads, c.dim, c.kv_rank);
            l.q_norm = to_f32(*m.dq_norm); l.kv_norm = to_f32(*m.dkv_norm);
        }
        if (module->has_mlp()) {
            l.norm2 = pack_norm(module->norm2);
            l.gate_up = interleave_rows(*module->gate, *module->up);
            l.down = module->down->raw_data();
        }
        layers_.push_back(std::move(l));
    }
    final_norm_ = pack_norm(owner_.final_norm(), owner_.logit_scale());   // logits = head (norm(x) * logit_scale)
    if (owner_.loop_step()) loop_step_ = to_f32(*owner_.loop_step());
    if (owner_.loop_in()) {   // "loop.in" [x; first] = loop_x_ x + loop_first_ first
        loop_x_ = owner_.loop_in()->narrow(1, 0, owner_.width());
        loop_first_ = owner_.loop_in()->narrow(1, owner_.width(), owner_.width());
    }
    synchronize(Device::cuda(device()));
    packed_version_ = version;
}

bool HybridPlan::shadows_for(Index rows) const {
    if (owner_.dtype() != DType::bf16 || rows <= 0) return false;
    const Index D = owner_.width();
    auto takes = [&](Index in, Index out) { return b200_linear_shadow_parts(rows, in, out) > 0; };
    if (D % 8 || !takes(D, owner_.vocabulary())) return false;
    for (std::size_t i = 0; i < layers_.size(); ++i) {
        const HybridLayer& module = *owner_.layers()[i];
        if (module.attention && !takes(D, layers_[i].attention_columns)) return false;
        if (!takes(D, layers_[i].wide_out) || !takes(layers_[i].inner, D)) return false;
        if (module.latent && !takes(module.latent->config().q_rank, module.latent->uq->size(0))) return false;
        if (module.has_mlp() && (!takes(D, 2 * module.gate->size(0)) || (owner_.design().form != LayerForm::parallel && !takes(module.gate->size(0), D))))
            return false;
        if (layers_[i].router.defined() && !takes(D, layers_[i].router.size(0))) return false;
    }
    return true;
}

void HybridPlan::grow(Tensor& t, Shape shape, DType dtype) {
    Index n = 1;
    for (const Index extent : shape) n *= extent;
    if (t.defined() && t.dtype() == dtype && t.device().index == device() && t.numel() >= n) return;
    synchronize(Device::cuda(device()));
    t = empty(std::move(shape), {dtype, Device::cuda(device())});
    ++epoch_;
}

b200_latent_args HybridPlan::latent_args(const Layer& layer, const LatentAttentionMixer& mixer, const HybridCache& cache, std::size_t run) const {
    const auto& c = mixer.config();
    b200_latent_args a{};
    a.heads = static_cast<int32_t>(c.heads); a.dim = static_cast<int32_t>(c.dim); a.rot_dim = static_cast<int32_t>(c.rot_dim);
    a.vdim = static_cast<int32_t>(c.vdim); a.kv_rank = static_cast<int32_t>(c.kv_rank); a.q_rank = static_cast<int32_t>(c.q_rank);
    a.rot_dims = static_cast<int32_t>(c.rot_dims);
    a.scale = static_cast<float>(c.scale); a.eps = owner_.eps();
    const auto& table = cache.rotary(c.rot_dims, c.rot_base);
    a.cosine = table.cosine.data<float>(); a.sine = table.sine.data<float>(); a.positions = static_cast<int32_t>(table.cosine.size(0));
    a.q_norm = layer.q_norm.data<float>(); a.kv_norm = layer.kv_norm.data<float>();
    a.cache = cache.run(run).latent;
    a.weight_dtype = code_of(owner_.dtype()); a.w_key = layer.w_key.raw_data(); a.w_value = layer.w_value;
    return a;
}

void HybridPlan::reserve(Index rows, Index max_length, const HybridCache& cache, const b200_rows& pass) {
    runtime::set_device(device());
    const Index D = owner_.width();
    const bool bf16 = owner_.dtype() == DType::bf16;
    Index wide = 0, inner = 0, channels = 0, y = 0, query = 0, absorbed = 0, latent = 0;
    std::size_t scratch = 0;
    for (std::size_t i = 0; i < owner_.runs().size(); ++i) {
        const auto index = static_cast<std::size_t>(owner_.runs()[i].layer);
        const HybridLayer& module = *owner_.layers()[index];
        wide = std::max(wide, layers_[index].wide_out);
        inner = std::max(inner, layers_[index].inner);
        if (module.has_mlp() && owner_.design().form != LayerForm::parallel) inner = std::max(inner, module.gate->size(0));
        if (module.lightning) {
            channels = std::max(channels, module.lightning->channels());
            y = std::max(y, module.lightning->inner());
        }
        if (module.delta) {
            channels = std::max(channels, module.delta->channels());
            y = std::max(y, module.delta->inner());
            continue;
        }
        if (module.attention) continue;   // reserve_attention
        if (module.state_space) {
            channels = std::max(channels, module.state_space->channels());
            y = std::max(y, module.state_space->inner());
        } else {
            const auto& c = module.latent->config();
            inner = std::max(inner, c.q_rank);
            query = std::max(query, c.heads * (c.dim + c.rot_dim));
            absorbed = std::max(absorbed, c.heads * (c.kv_rank + c.rot_dim));
            latent = std::max(latent, c.heads * c.kv_rank);
            const b200_latent_args a = latent_args(layers_[index], *module.latent, cache, i);
            scratch = std::max(scratch, b200_latent_scratch_bytes(&a, rows, pass.sequences, pass.max_count, static_cast<int32_t>(max_length)));
        }
    }
    grow(first_, {rows, D}, DType::f32);
    grow(h_, {rows, D}, DType::f32);
    grow(projected_, {rows, wide}, DType::f32);
    if (channels) { grow(mixed_, {rows, channels}, DType::f32); grow(y_, {rows, y}, DType::f32); }
    if (query) { grow(query_, {rows, query}, DType::f32); grow(absorbed_, {rows, absorbed}, DType::f32); grow(latent_out_, {rows, latent}, DType::f32); }
    if (bf16 && shadows_for(rows)) {
        grow(n_, rows, D);
        grow(i_, rows, inner);
        if (owner_.design().norm != NormKind::dynamic_tanh) {
            Index parts = 1;
            for (const auto& layer : layers_) parts = std::max<Index>(parts, b200_linear_shadow_parts(rows, layer.inner, D));
            if (owner_.loop_in()) parts = std::max<Index>(parts, b200_linear_shadow_parts(rows, D, D));
            grow(squares_, {parts, rows}, DType::f32);
        }
        if (owner_.loop_in()) grow(x_, rows, D);
    } else {
        grow(plain_, {rows, D}, DType::f32);
        grow(plain_inner_, {rows, inner}, DType::f32);
    }
    grow(scratch_, {static_cast<Index>(scratch / 4 + 1)}, DType::f32);
    if (owner_.loop_in()) { grow(joined_first_, {rows, D}, DType::f32); grow(entered_, {rows, D}, DType::f32); }
    if (norms_behind()) {
        grow(branch_, {rows, D}, DType::f32);
        Index outputs = 0;
        for (const auto& layer : layers_)
            if (layer.router.defined()) outputs = std::max(outputs, layer.router.size(0));
        if (outputs) grow(route_logits_, {rows, outputs}, DType::f32);
    }
    reserve_attention(rows, max_length, cache, pass);
}

void HybridPlan::linear(const float* x, Index rows, Index in, const void* w, Index out, b200_epilogue epilogue, const float* residual, float* y,
                        void* stream, const char* what) {
    runtime::check(b200_linear(x, rows, in, w, code_of(owner_.dtype()), out, nullptr, 0, 0.0, epilogue, residual, nullptr, y, stream), what);
    probe(0);
}

void HybridPlan::shadow(const Planes& x, Index rows, Index in, const void* w, Index out, b200_epilogue epilogue, const float* residual, float* y,
                        const Norm* next, Planes* to, void* stream, const char* what, Index to_column, Index to_stride, const b200_clamped_unit* unit) {
    b200_shadow_linear_args args{};
    args.x_hi = x.hi.raw_data();
    args.x_lo = owner_.activation_dtype() == DType::bf16 && rows >= 17 ? nullptr : x.lo.raw_data();
    args.rows = rows; args.in = in; args.weight = w; args.out = out;
    args.epilogue = epilogue; args.residual = residual; args.y = y; args.unit = unit;
    if (x.parts > 0) { args.sumsq_in = squares_.data<float>(); args.parts_in = static_cast<int32_t>(x.parts); args.eps = owner_.eps(); }
    b200_elementwise_norm norm{};
    if (to) {
        args.out_hi = static_cast<std::uint16_t*>(to->hi.mutable_data()) + to_column;
        args.out_lo = static_cast<std::uint16_t*>(to->lo.mutable_data()) + to_column;
        args.out_stride = to_stride;
        to->parts = 0;
    }
    if (next && next->rms) {
        args.out_norm_weight = next->weight.raw_data(); args.out_norm_dtype = B200_F32;
        args.sumsq_out = f32(squares_);
        to->parts = b200_linear_shadow_parts(rows, in, out);
    } else if (next) {
        norm = {next->alpha, next->weight.data<float>(), next->bias.data<float>()};
        args.out_norm = &norm;
    }
    runtime::check(b200_linear_shadow(&args, stream), what);
    probe(0);
}

// Planes of the rows under an RMS norm, whose factor the consumer applies.
void HybridPlan::planes_of(const float* x, Index rows, const Norm& norm, Planes& to, void* stream) {
    runtime::check(b200_shadow_from_rows(x, rows, owner_.width(), norm.weight.raw_data(), B200_F32, to.hi.mutable_data(), to.lo.mutable_data(),
                                         f32(squares_), stream), "norm");
    to.parts = 1;
    probe(2);
}

void HybridPlan::run(const Index* ids, const b200_rows& pass, HybridCache& cache, Index max_length, void* stream, std::vector<float>* trail) {
    ids_ = ids;
    if (norms_behind()) return run_sandwich(ids, pass, cache, max_length, stream, trail);
    const Index rows = pass.rows, D = owner_.width();
    const bool planes = shadows_for(rows);
    float *first = f32(first_), *h = f32(h_);
    const bool rms = owner_.design().norm != NormKind::dynamic_tanh;
    const auto& runs = owner_.runs();
    bool normed = false;   // the previous kernel has written this run's norm1
    auto embed = [&](const Norm* norm, Planes& to) {
        runtime::check(b200_embedding_shadow(owner_.embed().raw_data(), code_of(owner_.dtype()), ids, rows, owner_.vocabulary(), D,
                                             norm ? norm->weight.raw_data() : nullptr, B200_F32, first, to.hi.mutable_data(), to.lo.mutable_data(),
                                             f32(squares_), stream), "embedding");
        to.parts = norm ? 1 : 0;
        probe(2);
    };
    if (rms && planes) {
        if (owner_.loop_in()) embed(nullptr, x_);
        if (!owner_.loop_in() || !runs.front().begins_pass) {
            embed(&layers_[static_cast<std::size_t>(runs.front().layer)].norm1, n_);
            normed = true;
        }
    } else {
        runtime::check(b200_embedding_scaled(owner_.embed().raw_data(), code_of(owner_.dtype()), ids, rows, owner_.vocabulary(), D,
                                             static_cast<float>(owner_.embedding_scale()), first, stream), "embedding");
        probe(2);
    }
    if (owner_.loop_in()) {   // the embedding output's share of every pass's entry
        if (planes) shadow(x_, rows, D, loop_first_.raw_data(), D, B200_EPI_STORE, nullptr, f32(joined_first_), nullptr, nullptr, stream, "loop projection");
        else linear(first, rows, D, loop_first_.raw_data(), D, B200_EPI_STORE, nullptr, f32(joined_first_), stream, "loop projection");
    }
    if (grouped_) runtime::check_cuda(cudaMemsetAsync(counts_.mutable_data(), 0, counts_.nbytes(), static_cast<cudaStream_t>(stream)), "cudaMemsetAsync");
    const float* in = first;
    auto stand_alone_norm = [&](const float* x, const float* add_rows, const float* add_vector, float* sum, const Norm& n) {
        if (n.rms && planes) return planes_of(x, rows, n, n_, stream);
        if (n.rms) {
            runtime::check(b200_rms_norm(x, n.weight.raw_data(), B200_F32, rows, D, owner_.eps(), f32(plain_), stream), "norm");
        } else {
            const b200_elementwise_norm norm{n.alpha, n.weight.data<float>(), n.bias.data<float>()};
            runtime::check(b200_dynamic_tanh(x, add_rows, add_vector, rows, D, &norm, sum, planes ? nullptr : f32(plain_),
                                             planes ? n_.hi.mutable_data() : nullptr, planes ? n_.lo.mutable_data() : nullptr, stream), "norm");
        }
        probe(2);
    };
    // residual projection of inner rows
    auto residual_projection = [&](Index inner, const void* w, const float* residual, const After& after, const char* what) {
        if (planes) {
            shadow(i_, rows, inner, w, D, B200_EPI_RESIDUAL, residual, h, after.norm, after.norm ? &n_ : after.raw ? &x_ : nullptr, stream, what);
        } else {
            linear(f32(plain_inner_), rows, inner, w, D, B200_EPI_RESIDUAL, residual, h, stream, what);
            if (after.norm) stand_alone_norm(h, nullptr, nullptr, nullptr, *after.norm);
        }
        in = h;
    };
    for (std::size_t i = 0; i < runs.size(); ++i) {
        const LayerRun& r = runs[i];
        const HybridLayer& module = *owner_.layers()[static_cast<std::size_t>(r.layer)];
        const Layer& layer = layers_[static_cast<std::size_t>(r.layer)];
        if (r.begins_pass && owner_.loop_in()) {
            float* entered = f32(entered_);
            if (planes) {
                shadow(x_, rows, D, loop_x_.raw_data(), D, B200_EPI_RESIDUAL, f32(joined_first_), entered, &layer.norm1, &n_, stream, "loop projection");
            } else {
                linear(in, rows, D, loop_x_.raw_data(), D, B200_EPI_RESIDUAL, f32(joined_first_), entered, stream, "loop projection");
                stand_alone_norm(entered, nullptr, nullptr, nullptr, layer.norm1);
            }
            in = entered;
        } else if (r.begins_pass) {
            stand_alone_norm(in, r.pass > 0 ? first : nullptr, loop_step_.data<float>() + r.pass * D, h, layer.norm1);
            in = h;
        } else if (!normed) {
            stand_alone_norm(in, nullptr, nullptr, nullptr, layer.norm1);
        }
        const bool last = i + 1 == runs.size();
        // (where a pass begins next, something is added or projected before the norm)
        const After after_layer = last ? After{&final_norm_, false}
            : runs[i + 1].begins_pass ? After{nullptr, owner_.loop_in() != nullptr} : After{&layers_[static_cast<std::size_t>(runs[i + 1].layer)].norm1, false};
        normed = after_layer.norm != nullptr;
        if (module.attention) {
            const float* residual = run_parallel(i, in, pass, cache, max_length, stream);
            residual_projection(layer.inner, layer.out, residual, after_layer, "output projection");
            if (trail) keep_rows(rows, *trail);
            continue;
        }
        const After after_mixer = module.has_mlp() ? After{&layer.norm2, false} : after_layer;
        float* projected = f32(projected_);
        if (planes) shadow(n_, rows, D, layer.in, layer.wide_out, B200_EPI_STORE, nullptr, projected, nullptr, nullptr, stream, "mixer projection");
        else linear(f32(plain_), rows, D, layer.in, layer.wide_out, B200_EPI_STORE, nullptr, projected, stream, "mixer projection");
        void* inner_hi = planes ? i_.hi.mutable_data() : nullptr;
        void* inner_lo = planes ? i_.lo.mutable_data() : nullptr;
        float* inner_plain = planes ? nullptr : f32(plain_inner_);
        if (module.state_space) {
            const auto& c = module.state_space->config();
            b200_ssm_args a{};
            a.heads = static_cast<int32_t>(c.heads); a.vdim = static_cast<int32_t>(c.vdim); a.state = static_cast<int32_t>(c.state);
            a.groups = static_cast<int32_t>(c.groups); a.taps = static_cast<int32_t>(c.taps);
            a.conv_weight = layer.conv.data<float>(); a.conv_bias = layer.conv_bias.data<float>(); a.dt_bias = layer.dt_bias.data<float>();
            a.a_log = layer.a_log.data<float>(); a.d = layer.d.data<float>();
            a.conv_state = f32(cache.run(i).conv); a.ssm_state = f32(cache.run(i).state);
            a.projected = projected; a.mixed = f32(mixed_); a.y = f32(y_);
            runtime::check(b200_ssm_forward(&a, &pass, stream), "state-space recurrence");
            probe(1);
            runtime::check(b200_gated_group_norm(a.y, projected, layer.wide_out, layer.gated_norm.data<float>(), rows, layer.inner,
                                                 static_cast<int32_t>(c.norm_groups), owner_.eps(), inner_plain, inner_hi, inner_lo, stream), "gated norm");
            probe(2);
        } else {
            const auto& c = module.latent->config();
            const b200_latent_args a = latent_args(layer, *module.latent, cache, i);
            runtime::check(b200_latent_prepare(&a, &pass, projected, inner_plain, inner_hi, inner_lo, stream), "latent norms");
            probe(2);
            const Index query_out = c.heads * (c.dim + c.rot_dim);
            if (planes) shadow(i_, rows, c.q_rank, layer.uq, query_out, B200_EPI_STORE, nullptr, f32(query_), nullptr, nullptr, stream, "query up-projection");
            else linear(f32(plain_inner_), rows, c.q_rank, layer.uq, query_out, B200_EPI_STORE, nullptr, f32(query_), stream, "query up-projection");
            runtime::check(b200_latent_query(&a, &pass, f32(query_), f32(absorbed_), stream), "absorbed query");
            probe(0);
            runtime::check(b200_latent_attention(&a, &pass, f32(absorbed_), static_cast<int32_t>(max_length), scratch_.mutable_data(),
                                                 scratch_.nbytes(), f32(latent_out_), stream), "latent attention");
            probe(1);
            runtime::check(b200_latent_value(&a, rows, f32(latent_out_), projected + c.q_rank + c.kv_rank + c.rot_dim, layer.wide_out, inner_plain,
                                             inner_hi, inner_lo, stream), "value up-projection");
            probe(0);
        }
        residual_projection(layer.inner, layer.out, in, after_mixer, "output projection");
        if (module.has_mlp()) {
            const Index ff = module.gate->size(0);
            if (planes) shadow(n_, rows, D, layer.gate_up.raw_data(), 2 * ff, B200_EPI_SWIGLU, nullptr, nullptr, nullptr, &i_, stream, "gate/up projection");
            else linear(f32(plain_), rows, D, layer.gate_up.raw_data(), 2 * ff, B200_EPI_SWIGLU, nullptr, f32(plain_inner_), stream, "gate/up projection");
            residual_projection(ff, layer.down, in, after_layer, "down projection");
        }
        if (trail) keep_rows(rows, *trail);
    }
}

void HybridPlan::logits(Index rows, float* out, void* stream) {
    const Index D = owner_.width(), V = owner_.vocabulary();
    if (shadows_for(rows)) shadow(n_, rows, D, owner_.head().raw_data(), V, B200_EPI_STORE, nullptr, out, nullptr, nullptr, stream, "logits");
    else linear(f32(plain_), rows, D, owner_.head().raw_data(), V, B200_EPI_STORE, nullptr, out, stream, "logits");
    if (owner_.logit_softcap() > 0.0) runtime::check(b200_soft_cap(out, rows * V, static_cast<float>(owner_.logit_softcap()), stream), "logit cap");
}

void HybridPlan::logits_of(const std::int32_t* index, Index count, float* out, void* stream) {
    const Index D = owner_.width(), V = owner_.vocabulary();
    const bool planes = shadows_for(count);
    grow(picked_, {count, D}, DType::f32);
    if (planes) grow(p_, count, D);
    runtime::check(b200_gather_rows(f32(h_), index, count, D, f32(picked_), stream), "gather rows");
    if (final_norm_.rms && planes) {
        grow(squares_, {1, count}, DType::f32);
        planes_of(f32(picked_), count, final_norm_, p_, stream);
    } else if (final_norm_.rms) {
        runtime::check(b200_rms_norm(f32(picked_), final_norm_.weight.raw_data(), B200_F32, count, D, owner_.eps(), f32(picked_), stream), "final norm");
    } else {
        const b200_elementwise_norm norm{final_norm_.alpha, final_norm_.weight.data<float>(), final_norm_.bias.data<float>()};
        runtime::check(b200_dynamic_tanh(f32(picked_), nullptr, nullptr, count, D, &norm, nullptr, planes ? nullptr : f32(picked_),
                                         planes ? p_.hi.mutable_data() : nullptr, planes ? p_.lo.mutable_data() : nullptr, stream), "final norm");
    }
    if (planes) shadow(p_, count, D, owner_.head().raw_data(), V, B200_EPI_STORE, nullptr, out, nullptr, nullptr, stream, "logits");
    else linear(f32(picked_), count, D, owner_.head().raw_data(), V, B200_EPI_STORE, nullptr, out, stream, "logits");
    if (owner_.logit_softcap() > 0.0) runtime::check(b200_soft_cap(out, count * V, static_cast<float>(owner_.logit_softcap()), stream), "logit cap");
}

void HybridPlan::keep_rows(Index rows, std::vector<float>& trail) const {
    const auto count = static_cast<std::size_t>(rows * owner_.width()), at = trail.size();
    trail.resize(at + count);
    runtime::copy_bytes(trail.data() + at, Device::cpu(), f32(h_), Device::cuda(device()), count * sizeof(float));
}

void HybridPlan::advance(const b200_rows& pass, HybridCache& cache, void* stream) {
    if (owner_.pairs()) runtime::check(b200_rows_advance_tokens(&pass, ids_, cache.last_tokens(), stream), "advance");
    else runtime::check(b200_rows_advance(&pass, stream), "advance");
}


bool HybridPlan::prepare_choice(Index rows) {
    if (!shadows_for(rows)) return false;
    const Index parts = b200_linear_argmax_parts(rows, owner_.width(), owner_.vocabulary());
    if (parts <= 0) return false;
    grow(best_value_, {parts * rows}, DType::f32);
    grow(best_index_, {parts * rows}, DType::f32);   // int32 payload
    return true;
}

// (a cap on the logits keeps their order: the choice is made from the logits before it)
void HybridPlan::choose(Index rows, const TokenFeedback& f, void* stream) {
    const Index D = owner_.width(), V = owner_.vocabulary();
    b200_shadow_linear_args args{};
    args.x_hi = n_.hi.raw_data();
    args.x_lo = owner_.activation_dtype() == DType::bf16 && rows >= 17 ? nullptr : n_.lo.raw_data();
    if (n_.parts > 0) { args.sumsq_in = squares_.data<float>(); args.parts_in = static_cast<int32_t>(n_.parts); args.eps = owner_.eps(); }
    args.rows = rows; args.in = D; args.weight = owner_.head().raw_data(); args.out = V;
    args.epilogue = B200_EPI_ARGMAX;
    args.best_value = f32(best_value_);
    args.best_index = static_cast<std::int32_t*>(best_index_.mutable_data());
    runtime::check(b200_linear_shadow(&args, stream), "logits + argmax");
    probe(0);
    runtime::check(b200_argmax_finish(args.best_value, args.best_index, b200_linear_argmax_parts(rows, D, V), rows, f.next, f.ids, f.history,
                                      f.history_rows, f.counter, nullptr, 0, stream), "argmax merge");
    probe(2);
}

// [slot: S | first: S + 1 | sequence: rows], int32
b200_rows HybridPlan::PassMaps::describe(std::span<const Index> slots, std::span<const Index> counts, HybridCache& cache, int device) {
    const std::size_t S = slots.size();
    Index rows = 0, longest = 0;
    for (const Index n : counts) { rows += n; longest = std::max(longest, n); }
    const std::size_t words = 2 * S + 1 + static_cast<std::size_t>(rows), bytes = words * sizeof(std::int32_t);
    const Device where = Device::cuda(device);
    if (!block.defined() || block.nbytes() < bytes) {
        synchronize(where);
        block = empty({static_cast<Index>(words)}, {DType::f32, where});
        staging = std::make_shared<runtime::Storage>(bytes, Device::cpu(), true);
    }
    auto* words_host = static_cast<std::int32_t*>(staging->data);
    Index at = 0;
    for (std::size_t s = 0; s < S; ++s) {
        words_host[s] = static_cast<std::int32_t>(slots[s]);
        words_host[S + s] = static_cast<std::int32_t>(at);
        for (Index i = 0; i < counts[s]; ++i) words_host[2 * S + 1 + static_cast<std::size_t>(at + i)] = static_cast<std::int32_t>(s);
        at += counts[s];
    }
    words_host[2 * S] = static_cast<std::int32_t>(at);
    runtime::check_cuda(cudaMemcpyAsync(block.mutable_data(), words_host, bytes, cudaMemcpyHostToDevice, cuda_stream(device)), "cudaMemcpyAsync");
    const auto* base = static_cast<const std::int32_t*>(block.raw_data());
    b200_rows pass{};
    pass.rows = rows; pass.sequences = static_cast<int32_t>(S); pass.max_count = static_cast<int32_t>(longest);
    pass.slot = base; pass.first = base + S; pass.sequence = base + 2 * S + 1; pass.lengths = cache.lengths();
    return pass;
}

// ---- passes -------------------------------------------------------------------------------------------------
namespace {
void check_pass(const HybridDecoder& model, const HybridCache& cache, std::span<const PassEntry> entries) {
    std::vector<char> seen(static_cast<std::size_t>(cache.slots()), 0);
    for (const auto& e : entries) {
        const Index length = cache.length(e.slot);   // range check
        if (seen[static_cast<std::size_t>(e.slot)]++) throw std::invalid_argument("a slot appears twice in one pass");
        if (e.tokens.empty()) throw std::invalid_argument("every entry of a pass needs at least one token");
        if (static_cast<Index>(e.tokens.size()) > cache.capacity() - length) throw std::invalid_argument("the pass exceeds the cache's capacity");
        for (const Index id : e.tokens)
            if (id < 0 || id >= model.vocabulary()) throw std::out_of_range("embedding index out of range");
        for (const Index w : e.want)
            if (w < 0 || w >= static_cast<Index>(e.tokens.size())) throw std::out_of_range("a wanted place lies outside the entry's tokens");
    }
}
}  // namespace

void HybridDecoder::pass(HybridCache& cache, std::span<const PassEntry> entries, float* logits, std::vector<float>* trail) {
    if (entries.empty()) return;
    check_pass(*this, cache, entries);   // everything that can fail for the caller's sake fails before the first launch
    auto& p = plan();
    p.refresh();
    p.set_user(nullptr);
    const int device = p.device();
    if (device != cache.device()) throw std::invalid_argument("the cache lives on another device");
    runtime::set_device(device);
    cudaStream_t stream = cuda_stream(device);
    const Device where = Device::cuda(device);
    // Where each entry's wanted rows go in the result.
    std::vector<Index> result_at(entries.size());
    Index wanted_total = 0;
    for (std::size_t e = 0; e < entries.size(); ++e) { result_at[e] = wanted_total; wanted_total += static_cast<Index>(entries[e].want.size()); }
    if (wanted_total && !logits) throw std::invalid_argument("wanted logits need a result buffer");
    // Cut into passes of at most kPassRows rows: a sequence's tokens stay in order, so the cuts change nothing but rounding.
    std::vector<Index> done(entries.size(), 0);
    std::size_t next = 0;
    while (next < entries.size()) {
        std::vector<Index> slots, counts, ids;
        std::vector<std::int32_t> picked;
        std::vector<Index> picked_to;
        Index rows = 0, max_length = 0;
        std::vector<std::size_t> members;
        for (std::size_t e = next; e < entries.size() && rows < kPassRows; ++e) {
            const auto& entry = entries[e];
            const Index take = std::min<Index>(static_cast<Index>(entry.tokens.size()) - done[e], kPassRows - rows);
            for (std::size_t w = 0; w < entry.want.size(); ++w)
                if (entry.want[w] >= done[e] && entry.want[w] < done[e] + take) {
                    picked.push_back(static_cast<std::int32_t>(rows + entry.want[w] - done[e]));
                    picked_to.push_back(result_at[e] + static_cast<Index>(w));
                }
            ids.insert(ids.end(), entry.tokens.begin() + done[e], entry.tokens.begin() + done[e] + take);
            slots.push_back(entry.slot);
            counts.push_back(take);
            members.push_back(e);
            rows += take;
            max_length = std::max(max_length, cache.length(entry.slot) + take);
        }
        const Tensor device_ids = detail::from_host(ids.data(), {rows}, DType::i64, false, where);
        const b200_rows description = p.maps.describe(slots, counts, cache, device);
        p.reserve(rows, max_length, cache, description);
        p.run(device_ids.data<Index>(), description, cache, max_length, stream, trail);
        p.advance(description, cache, stream);
        for (std::size_t m = 0; m < members.size(); ++m) { cache.commit(slots[m], counts[m]); done[members[m]] += counts[m]; }
        while (next < entries.size() && done[next] == static_cast<Index>(entries[next].tokens.size())) ++next;
        if (!picked.empty()) {
            const Index n = static_cast<Index>(picked.size());
            Tensor index = empty({n}, {DType::f32, where});
            runtime::copy_bytes(index.mutable_data(), where, picked.data(), Device::cpu(), picked.size() * sizeof(std::int32_t));
            Tensor out = empty({n, vocab_}, {DType::f32, where});
            p.logits_of(static_cast<const std::int32_t*>(index.raw_data()), n, f32(out), stream);
            const Tensor host = out.to(Device::cpu());
            for (Index i = 0; i < n; ++i)
                std::copy_n(host.data<float>() + i * vocab_, vocab_, logits + picked_to[static_cast<std::size_t>(i)] * vocab_);
        }
        synchronize(where);   // the pass's arrays are reused
    }
    std::int32_t status = 0;
    runtime::check(b200_take_device_status(device, stream, &status), "device status");
    if (status) throw std::runtime_error("a kernel of the pass gave up a bounded wait or met an invalid id (status " + std::to_string(status) + ")");
}

Tensor HybridDecoder::forward(const Tensor& input) {
    if (input.dtype() != DType::i64 || input.ndim() != 2) throw std::invalid_argument("HybridDecoder expects int64 ids [batch, length]");
    const Tensor ids = input.to(Device::cpu());
    const Index batch = ids.size(0), length = ids.size(1);
    Tensor host = empty({batch, length, vocab_}, {DType::f32, Device::cpu()});
    if (batch * length > 0) {
        HybridCache cache(*this, batch, length);
        std::vector<Index> all(static_cast<std::size_t>(length));
        for (Index i = 0; i < length; ++i) all[static_cast<std::size_t>(i)] = i;
        std::vector<PassEntry> entries;
        for (Index b = 0; b < batch; ++b) entries.push_back({b, {ids.data<Index>() + b * length, static_cast<std::size_t>(length)}, all});
        pass(cache, entries, f32(host));
    }
    return host.to(embed_->device());
}

// ---- generation ---------------------------------------------------------------------------------------------
namespace {

class HybridTokenModel : public TokenModel {
public:
    HybridTokenModel(std::shared_ptr<HybridDecoder> model, std::shared_ptr<HybridCache> cache) : model_(std::move(model)), cache_(std::move(cache)) {
        if (!model_ || !cache_) throw std::invalid_argument("generation needs a model and a cache");
        if (model_->embed().device().type != DeviceType::cuda || model_->embed().device().index != cache_->device())
            throw std::invalid_argument("generation: model and cache must live on one CUDA device");
    }
    int device() const override { return cache_->device(); }
    Index vocabulary() const override { return model_->vocabulary(); }
    Index outputs() const override { return model_->vocabulary(); }
    std::uint64_t version() const override { return model_->version(); }
    void refresh() override { model_->plan().refresh(); }
    void validate(Index batch, Index length) override {
        if (batch > cache_->slots()) throw std::invalid_argument("the cache has fewer slots than the batch has sequences");
        for (Index b = 0; b < batch; ++b)
            if (length > cache_->capacity() - cache_->length(b)) throw std::invalid_argument("the step exceeds the cache's capacity");
    }
    std::uint64_t buffer_epoch() const override { return model_->plan().buffer_epoch() + maps_epoch_; }
    void prefill(const Tensor& prompt, std::span<const Index> lengths, float* logits) override {
        const Index batch = prompt.size(0), P = prompt.size(1), V = model_->vocabulary();
        const Tensor ids = prompt.to(Device::cpu());
        std::vector<PassEntry> entries;
        std::vector<Index> last(static_cast<std::size_t>(batch));
        for (Index b = 0; b < batch; ++b) {
            const Index n = lengths.empty() ? P : lengths[static_cast<std::size_t>(b)];
            last[static_cast<std::size_t>(b)] = n - 1;
            entries.push_back({b, {ids.data<Index>() + b * P, static_cast<std::size_t>(n)}, {&last[static_cast<std::size_t>(b)], 1}});
        }
        Tensor host = empty({batch, V}, {DType::f32, Device::cpu()});
        model_->pass(*cache_, entries, f32(host));
        runtime::copy_bytes(logits, Device::cuda(device()), host.raw_data(), Device::cpu(), host.nbytes());
    }
    bool prepare_step(Index batch) override {
        if (maps_batch_ != batch) {
            std::vector<Index> slots(static_cast<std::size_t>(batch)), counts(static_cast<std::size_t>(batch), 1);
            for (Index b = 0; b < batch; ++b) slots[static_cast<std::size_t>(b)] = b;
            pass_ = maps_.describe(slots, counts, *cache_, device());
            maps_batch_ = batch;
            ++maps_epoch_;
        }
        auto& plan = model_->plan();
        plan.reserve(batch, cache_->capacity(), *cache_, pass_);
        return plan.prepare_choice(batch);
    }
    void step(const Index* ids, Index, void* stream) override { model_->plan().run(ids, pass_, *cache_, cache_->capacity(), stream); }
    void advance(Index, void* stream) override {
        model_->plan().advance(pass_, *cache_, stream);
        probe(2);
    }
    void logits(Index batch, float* out, void* stream) override { model_->plan().logits(batch, out, stream); }
    void choose(Index batch, const TokenFeedback& feedback, void* stream) override {
        advance(batch, stream);
        model_->plan().choose(batch, feedback, stream);
    }
    void commit(Index steps) override { for (Index b = 0; b < maps_batch_; ++b) cache_->commit(b, steps); }
    void set_user(const void* user) override { model_->plan().set_user(user); }
    const void* user() const override { return model_->plan().user(); }

private:
    std::shared_ptr<HybridDecoder> model_;
    std::shared_ptr<HybridCache> cache_;
    HybridPlan::PassMaps maps_;
    b200_rows pass_{};
    Index maps_batch_ = 0;
    std::uint64_t maps_epoch_ = 0;
};

}  // namespace

std::unique_ptr<TokenModel> make_token_model(std::shared_ptr<HybridDecoder> model, std::shared_ptr<HybridCache> cache) {
    return std::make_unique<HybridTokenModel>(std::move(model), std::move(cache));
}

}  // namespace dl::nn
