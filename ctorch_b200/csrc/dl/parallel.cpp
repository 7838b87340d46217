// Grouped-query attention and mixtures of experts of the configured decoders, and their parallel layers: attention and a feed-forward or a
// mixture on one norm (see hybrid.h).
#include "dl/hybrid_plan.h"

#include <algorithm>
#include <stdexcept>

namespace dl::nn {

namespace {
// Up to this many rows the units of a dense feed-forward are projected together with q, k, v and g and activated beside the norms of
// the heads (a launch less); longer passes project them on their own, where the epilogue activates them without a round trip.
constexpr Index kRowsBeside = 128;

Index round_up_8(Index n) { return (n + 7) & ~static_cast<Index>(7); }
}  // namespace

// ---- modules ------------------------------------------------------------------------------------------------
GroupedAttentionMixer::GroupedAttentionMixer(Index width, const GroupedAttentionConfig& c, TensorOptions options) : config_(c) {
    const AttentionKind& kind = c.kind;
    if (c.heads % c.kv_heads) throw std::invalid_argument("grouped attention: heads must be a multiple of kv_heads");
    if (c.rot_dims % 2 || c.rot_dims > c.dim) throw std::invalid_argument("grouped attention: rotated dimensions must be even and at most dim");
    if (kind.keys_as_values && c.vdim != c.dim) throw std::invalid_argument("grouped attention: values that are the keys must have their size");
    if ((c.chunk > 0 || c.window > 0) && !own_keys()) throw std::invalid_argument("grouped attention: chunks and windows need keys of the layer itself");
    if (c.keep > 0 && c.pool > 0) throw std::invalid_argument("grouped attention: kept first positions are not combined with pooled blocks");
    q = &register_parameter("q", host_zeros({c.heads * c.dim, width}, options));
    if (kind.bias) q_bias = &register_parameter("q.b", host_zeros({c.heads * c.dim}, options));
    if (own_keys()) {
        k = &register_parameter("k", host_zeros({c.kv_heads * c.dim, width}, options));
        if (kind.bias) k_bias = &register_parameter("k.b", host_zeros({c.kv_heads * c.dim}, options));
        if (!kind.keys_as_values) v = &register_parameter("v", host_zeros({c.kv_heads * c.vdim, width}, options));
    }
    if (kind.norm == B200_HEAD_NORM_PROJECTION || (kind.norm == B200_HEAD_NORM_HEAD && kind.head_weights)) {
        const bool per_head = kind.norm == B200_HEAD_NORM_HEAD;
        q_norm = &register_parameter("q.norm", ones({per_head ? c.dim : c.heads * c.dim}, options));
        if (own_keys()) k_norm = &register_parameter("k.norm", ones({per_head ? c.dim : c.kv_heads * c.dim}, options));
    }
    if (kind.sink == Sink::learned) sink = &register_parameter("sink", host_zeros({c.heads}, options));
    if (kind.gate != OutputGate::none) gate = &register_parameter("g", host_zeros({kind.gate == OutputGate::head ? c.heads : c.heads * c.vdim, width}, options));
    if (kind.talk) talk = &register_parameter("talk", host_zeros({c.heads, c.heads}, options));
    out = &register_parameter("o", host_zeros({width, c.heads * c.vdim}, options));
}
Index GroupedAttentionMixer::columns() const {
    Index count = 0;
    for (const Tensor* t : {q, k, v, gate})
        if (t) count += t->size(0);
    return count;
}

MixtureOfExperts::MixtureOfExperts(Index width, const MixtureConfig& c, TensorOptions options) : config_(c) {
    if (c.identity < 0) throw std::invalid_argument("mixture of experts: a negative number of identity experts");
    if (c.top > c.outputs()) throw std::invalid_argument("mixture of experts: 'top' exceeds the number of experts");
    if (c.outputs() > B200_MAX_EXPERTS) throw std::invalid_argument("mixture of experts: more than " + std::to_string(B200_MAX_EXPERTS) + " experts");
    for (Index e = 0; e < c.experts; ++e) {
        const std::string name = "e" + std::to_string(e);
        if (c.kind.gated) gate.push_back(&register_parameter(name + ".gate", host_zeros({c.ff, width}, options)));
        up.push_back(&register_parameter(name + ".up", host_zeros({c.ff, width}, options)));
        down.push_back(&register_parameter(name + ".down", host_zeros({width, c.ff}, options)));
    }
    router = &register_parameter("router", host_zeros({c.outputs(), width}, options));
    if (c.kind.bias) bias = &register_parameter("router.b", host_zeros({c.outputs()}, options));
    if (c.kind.correction) correction = &register_parameter("correction", host_zeros({c.outputs()}, options));
    if (c.shared_ff > 0) {
        if (c.kind.gated) throw std::invalid_argument("mixture of experts: a shared expert is not combined with gated experts");
        shared_up = &register_parameter("shared.up", host_zeros({c.shared_ff, width}, options));
        shared_down = &register_parameter("shared.down", host_zeros({width, c.shared_ff}, options));
    }
}

// ---- plan ---------------------------------------------------------------------------------------------------
void HybridPlan::pack_attention(const GroupedAttentionMixer& m, Layer& l) const {
    if (m.q_norm) l.q_norm = to_f32(*m.q_norm);
    if (m.k_norm) l.kv_norm = to_f32(*m.k_norm);
    if (m.q_bias) l.q_bias = to_f32(*m.q_bias);
    if (m.k_bias) l.k_bias = to_f32(*m.k_bias);
    if (m.sink) l.sink = to_f32(*m.sink);
    else if (m.config().kind.sink == Sink::zero) l.sink = zeros({m.config().heads}, {DType::f32, m.q->device()});
    if (m.talk) l.talk = to_f32(*m.talk);
}

void HybridPlan::pack_experts(const MixtureOfExperts& e, Layer& l) const {
    std::vector<Tensor> ups, downs;
    for (std::size_t i = 0; i < e.up.size(); ++i) ups.push_back(e.gate.empty() ? *e.up[i] : interleave_rows(*e.gate[i], *e.up[i]));
    for (const Tensor* t : e.down) downs.push_back(*t);
    l.experts_up = concat_rows(ups);
    l.experts_down = concat_rows(downs);
    if (e.correction) l.correction = to_f32(*e.correction);
    if (e.bias) l.router_bias = to_f32(*e.bias);
}

void HybridPlan::pack_parallel(const HybridLayer& module, Layer& l) const {
    const GroupedAttentionMixer& m = *module.attention;
    const Index D = owner_.width();
    const TensorOptions options{owner_.dtype(), m.q->device()};
    std::vector<Tensor> rows{*m.q, *m.k, *m.v, *m.gate}, columns{*m.out};
    Index count = m.columns();
    auto pad = [&] {   // sections of a projected row start at multiples of eight
        if (count % 8) rows.push_back(zeros({round_up_8(count) - count, D}, options));
        count = round_up_8(count);
    };
    pad();
    l.attention_columns = count;
    if (module.has_mlp()) {
        l.unit_column = count;
        l.units = module.gate->size(0);
        rows.push_back(interleave_rows(*module.gate, *module.up));
        columns.push_back(*module.down);
        count += 2 * l.units;
        pad();
    } else if (module.mixture) {
        const MixtureOfExperts& e = *module.mixture;
        l.router_column = count;
        rows.push_back(*e.router);
        count += e.config().experts;
        pad();
        if (e.shared_up) {
            l.unit_column = count;
            l.units = e.config().shared_ff;
            rows.push_back(*e.shared_up);
            columns.push_back(*e.shared_down);
            count += l.units;
            pad();
        }
        pack_experts(e, l);
    }
    l.wide = concat_rows(rows);
    l.in = l.wide.raw_data();
    l.wide_out = count;
    l.attended = m.out->size(1);
    l.joint = columns.size() == 1 ? columns.front() : concat_columns(columns);
    l.out = l.joint.raw_data();
    l.inner = l.attended + l.units;
    pack_attention(m, l);
}

bool HybridPlan::units_beside(const HybridLayer& module, Index rows, bool planes) const { return !module.has_mlp() || !planes || rows <= kRowsBeside; }

b200_chunk_args HybridPlan::chunk_args(const Layer& layer, const HybridLayer& module, const HybridCache& cache, std::size_t run, Index stride) const {
    const auto& c = module.attention->config();
    const HybridCache::Run& r = cache.run(static_cast<std::size_t>(owner_.runs()[run].keys_run));
    auto vector = [](const Tensor& t) { return t.defined() ? t.data<float>() : nullptr; };
    auto workspace = [](const Tensor& t) { return t.defined() ? t.mutable_data() : nullptr; };
    b200_chunk_args a{};
    a.heads = static_cast<int32_t>(c.heads); a.kv_heads = static_cast<int32_t>(c.kv_heads); a.dim = static_cast<int32_t>(c.dim);
    a.vdim = static_cast<int32_t>(c.vdim); a.rot_dims = static_cast<int32_t>(c.rot_dims);
    a.slots = static_cast<int32_t>(cache.slots());
    // (no position reaches a chunk that is longer than the cache)
    a.chunk = static_cast<int32_t>(c.chunk > cache.capacity() ? 0 : c.chunk); a.entries = static_cast<int32_t>(r.entries);
    a.scale = static_cast<float>(c.scale); a.eps = owner_.eps();
    if (c.rot_dims > 0) {
        const auto& table = cache.rotary(c.rot_dims, c.rot_base, c.rot_factor);
        a.cosine = table.cosine.data<float>(); a.sine = table.sine.data<float>(); a.positions = static_cast<int32_t>(table.cosine.size(0));
    }
    a.q_norm = vector(layer.q_norm); a.k_norm = vector(layer.kv_norm); a.q_bias = vector(layer.q_bias); a.k_bias = vector(layer.k_bias);
    a.sink = vector(layer.sink);
    a.norm = c.kind.norm; a.rotate_pairs = c.kind.rotate_pairs; a.keys_as_values = c.kind.keys_as_values; a.keys_elsewhere = !module.attention->own_keys();
    a.no_gate = c.kind.gate != OutputGate::head; a.gate_values = c.kind.gate == OutputGate::value; a.softcap = static_cast<float>(c.softcap);
    a.scaled = 1; a.out_scale = static_cast<float>(module.attention_scale);
    a.window = static_cast<int32_t>(r.window); a.keep = static_cast<int32_t>(r.keep); a.pool = static_cast<int32_t>(r.pools);
    a.pool_state = r.pool.defined() ? f32(r.pool) : nullptr;
    a.norm_values = c.kind.norm_values; a.talk = vector(layer.talk);
    a.dtype = code_of(owner_.dtype());
    a.key_cache = r.key.mutable_data(); a.value_cache = r.value.mutable_data();
    a.projected = projected_.data<float>(); a.stride = stride;
    a.query = chunk_query_.mutable_data(); a.key = workspace(chunk_key_); a.value = workspace(chunk_value_);
    return a;
}

b200_experts HybridPlan::expert_args(const Layer& layer, const MixtureOfExperts& mixture, Index rows) const {
    const auto& c = mixture.config();
    b200_experts a{};
    a.experts = static_cast<int32_t>(c.experts); a.top = static_cast<int32_t>(c.top);
    a.rows = rows; a.in = owner_.width(); a.ff = c.ff;
    a.weight_dtype = code_of(owner_.dtype());
    a.up = layer.experts_up.raw_data(); a.down = layer.experts_down.raw_data();
    a.chosen = static_cast<const std::int32_t*>(chosen_.raw_data()); a.weight = score_.data<float>();
    if (shadows_for(rows)) {
        a.x_hi = n_.hi.raw_data(); a.x_lo = n_.lo.raw_data();
        a.sumsq_in = squares_.data<float>(); a.parts_in = static_cast<int32_t>(n_.parts);
    } else {
        a.x = f32(plain_);
    }
    a.eps = owner_.eps();
    a.gated = c.kind.gated; a.weigh_results = c.kind.weigh_results; a.identity = static_cast<int32_t>(c.identity);
    a.residual = f32(h_); a.y = f32(h_);
    return a;
}

void HybridPlan::reserve_attention(Index rows, Index max_length, const HybridCache& cache, const b200_rows& pass) {
    grouped_ = false;
    Index query = 0, key = 0, value = 0, slots = 0, act = 0, most_experts = 0;
    for (const auto& module : owner_.layers()) {
        if (module->attention) {
            const auto& c = module->attention->config();
            query = std::max(query, c.heads * c.dim);
            if (c.chunk > 0 || c.window > 0) {   // without either the rows go into the slots at once
                key = std::max(key, c.kv_heads * c.dim);
                value = std::max(value, c.kv_heads * c.vdim);
            }
        }
        if (module->mixture) {
            const auto& c = module->mixture->config();
            slots = std::max(slots, c.top);
            act = std::max(act, c.top * c.ff);
            most_experts = std::max(most_experts, c.experts);
        }
    }
    if (query) grow(chunk_query_, {rows, query}, owner_.dtype());
    if (key) { grow(chunk_key_, {rows, key}, owner_.dtype()); grow(chunk_value_, {rows, value}, owner_.dtype()); }
    if (slots) {
        grow(chosen_, {rows, slots}, DType::f32);   // int32 payload
        grow(rank_, {rows, slots}, DType::f32);
        grow(score_, {rows, slots}, DType::f32);
        grow(counts_, {static_cast<Index>(owner_.runs().size()), most_experts}, DType::f32);
    }
    std::size_t scratch = 0, grouped = 0;
    bool streamed = false;
    for (std::size_t i = 0; i < owner_.runs().size(); ++i) {
        const auto index = static_cast<std::size_t>(owner_.runs()[i].layer);
        const HybridLayer& module = *owner_.layers()[index];
        if (module.attention) {
            const b200_chunk_args a = chunk_args(layers_[index], module, cache, i, layers_[index].wide_out);
            scratch = std::max(scratch, b200_chunk_scratch_bytes(&a, rows, pass.sequences, pass.max_count, static_cast<int32_t>(max_length)));
        }
        if (module.mixture) {
            const b200_experts a = expert_args(layers_[index], *module.mixture, rows);
            if (b200_experts_takes_grouped(&a)) grouped = std::max(grouped, b200_experts_grouped_bytes(&a));
            else streamed = true;
        }
    }
    if (scratch) grow(scratch_, {static_cast<Index>(scratch / 4 + 1)}, DType::f32);
    if (grouped) grow(expert_scratch_, {static_cast<Index>(grouped / 4)}, DType::f32);
    if (streamed) grow(expert_act_, {rows, act}, DType::f32);
    grouped_ = grouped > 0;
}

const float* HybridPlan::run_parallel(std::size_t run, const float* in, const b200_rows& pass, HybridCache& cache, Index max_length, void* stream) {
    const LayerRun& r = owner_.runs()[run];
    const HybridLayer& module = *owner_.layers()[static_cast<std::size_t>(r.layer)];
    const Layer& layer = layers_[static_cast<std::size_t>(r.layer)];
    const Index rows = pass.rows, D = owner_.width();
    const bool planes = shadows_for(rows), beside = units_beside(module, rows, planes);
    const Index stride = beside ? layer.wide_out : layer.attention_columns;
    float* projected = f32(projected_);
    if (planes) shadow(n_, rows, D, layer.in, stride, B200_EPI_STORE, nullptr, projected, nullptr, nullptr, stream, "mixer projection");
    else linear(f32(plain_), rows, D, layer.in, stride, B200_EPI_STORE, nullptr, projected, stream, "mixer projection");
    if (!beside) {
        const auto* gate_up = static_cast<const std::uint16_t*>(layer.in) + layer.unit_column * D;
        shadow(n_, rows, D, gate_up, 2 * layer.units, B200_EPI_SWIGLU, nullptr, nullptr, nullptr, &i_, stream, "gate/up projection", layer.attended, layer.inner);
    }

    const b200_chunk_args a = chunk_args(layer, module, cache, run, stride);
    float* inner_plain = planes ? nullptr : f32(plain_inner_);
    auto* inner_hi = planes ? static_cast<std::uint16_t*>(i_.hi.mutable_data()) : nullptr;
    auto* inner_lo = planes ? static_cast<std::uint16_t*>(i_.lo.mutable_data()) : nullptr;
    b200_units units{};
    if (beside && layer.units > 0) {
        units.kind = module.has_mlp() ? 1 : 2;
        units.column = layer.unit_column; units.count = layer.units; units.out_stride = layer.inner;
        if (planes) { units.out_hi = inner_hi + layer.attended; units.out_lo = inner_lo + layer.attended; }
        else units.out = inner_plain + layer.attended;
    }
    b200_route route{};
    b200_experts experts{};
    bool grouped = false;
    if (module.mixture) {
        experts = expert_args(layer, *module.mixture, rows);
        experts.residual = in;
        grouped = b200_experts_takes_grouped(&experts) != 0;
        route.experts = experts.experts; route.top = experts.top; route.column = layer.router_column;
        route.chosen = static_cast<std::int32_t*>(chosen_.mutable_data()); route.weight = f32(score_);
        if (grouped) {
            route.rank = static_cast<std::int32_t*>(rank_.mutable_data());
            route.counts = static_cast<std::int32_t*>(counts_.mutable_data()) + static_cast<Index>(run) * (counts_.numel() / static_cast<Index>(owner_.runs().size()));
        }
    }
    runtime::check(b200_chunk_prepare(&a, &pass, &units, &route, stream), "attention norms");
    probe(2);
    runtime::check(b200_chunk_attention(&a, &pass, static_cast<int32_t>(max_length), scratch_.mutable_data(), scratch_.nbytes(), inner_plain, inner_hi, inner_lo,
                                        layer.inner, stream), "grouped attention");
    probe(1);
    if (!module.mixture) return in;
    if (grouped) runtime::check(b200_experts_grouped(&experts, route.rank, route.counts, expert_scratch_.mutable_data(), expert_scratch_.nbytes(), stream), "experts");
    else runtime::check(b200_experts_streamed(&experts, f32(expert_act_), stream), "experts");
    probe(0);
    return f32(h_);
}

}  // namespace dl::nn
