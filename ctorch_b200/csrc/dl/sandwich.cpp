// Layers of the configured decoders with a norm behind every sublayer, and one before it or none: attention alone or side by side with
// lightning attention or the delta rule (delta.cpp), clamped gated units or a mixture of gated experts, and the embedding of token pairs
// (see hybrid.h).
#include "dl/hybrid_plan.h"

#include <algorithm>
#include <stdexcept>

namespace dl::nn {

namespace {
Index round_up_8(Index n) { return (n + 7) & ~static_cast<Index>(7); }
}  // namespace

// ---- modules ------------------------------------------------------------------------------------------------
LightningMixer::LightningMixer(Index width, const LightningConfig& c, TensorOptions options) : config_(c) {
    if (static_cast<Index>(c.decay.size()) != c.heads) throw std::invalid_argument("lightning attention: 'decay' must have one number per head");
    if (c.dim > B200_SSM_MAX_STATE) throw std::invalid_argument("lightning attention: 'dim' exceeds " + std::to_string(B200_SSM_MAX_STATE));
    q = &register_parameter("q", host_zeros({c.heads * c.dim, width}, options));
    k = &register_parameter("k", host_zeros({c.heads * c.dim, width}, options));
    v = &register_parameter("v", host_zeros({inner(), width}, options));
    gate = &register_parameter("g", host_zeros({inner(), width}, options));
    norm = &register_parameter("norm", ones({inner()}, options));
    out = &register_parameter("o", host_zeros({width, inner()}, options));
}

SideBySideMixer::SideBySideMixer(Index width, const GroupedAttentionConfig& l, const LightningConfig& r, double scale_left, double scale_right,
                                 TensorOptions options)
    : left_scale(scale_left), right_scale(scale_right) {
    left = add_module<GroupedAttentionMixer>("left", width, l, options);
    right = add_module<LightningMixer>("right", width, r, options);
}

// ---- plan ---------------------------------------------------------------------------------------------------
void HybridPlan::pack_sandwich(const HybridLayer& module, Layer& l) const {
    const Index D = owner_.width();
    const TensorOptions options{owner_.dtype(), owner_.embed().device()};
    // (what a sublayer adds is multiplied by the factor of the residual: in the weight of the norm behind it)
    l.after1 = pack_norm(module.after1, owner_.residual_factor());
    if (module.after2.weight) l.after2 = pack_norm(module.after2, owner_.residual_factor());
    if (module.norm2.weight) l.norm2 = pack_norm(module.norm2);
    if (module.has_mlp()) {
        l.gate_up = interleave_rows(*module.gate, *module.up);
        l.down = module.down->raw_data();
        l.unit = {static_cast<float>(owner_.design().unit_slope), static_cast<float>(module.unit_limit)};
    } else if (module.mixture) {
        const Tensor& router = *module.mixture->router;
        const Index outputs = router.size(0), padded = round_up_8(outputs);
        l.router = router;
        if (padded > outputs) {
            const Tensor parts[2] = {router, zeros({padded - outputs, D}, options)};
            l.router = concat_rows(parts);
        }
        pack_experts(*module.mixture, l);
    }
    if (module.delta) return pack_delta(*module.delta, l);
    const GroupedAttentionMixer& m = *module.attention;
    std::vector<Tensor> rows, columns{*m.out};
    for (const Tensor* t : {m.q, m.k, m.v, m.gate})
        if (t) rows.push_back(*t);
    Index count = m.columns();
    auto pad = [&] {   // sections of a projected row start at multiples of eight
        if (count % 8) rows.push_back(zeros({round_up_8(count) - count, D}, options));
        count = round_up_8(count);
    };
    pad();
    l.attention_columns = count;
    if (module.lightning) {   // in the order of the recurrence's columns
        const LightningMixer& r = *module.lightning;
        l.lightning_column = count;
        for (const Tensor* t : {r.gate, r.v, r.k, r.q}) rows.push_back(*t);
        columns.push_back(*r.out);
        count += r.inner() + r.channels();
        pad();
        Tensor decay = empty({r.config().heads}, {DType::f32, Device::cpu()});
        for (Index h = 0; h < r.config().heads; ++h) f32(decay)[h] = static_cast<float>(r.config().decay[static_cast<std::size_t>(h)]);
        l.decay = decay.to(m.q->device());
        l.right_norm = to_f32(*r.norm);
    }
    l.wide = rows.size() == 1 ? rows.front() : concat_rows(rows);
    l.in = l.wide.raw_data();
    l.wide_out = count;
    l.joint = columns.size() == 1 ? columns.front() : concat_columns(columns);
    l.out = l.joint.raw_data();
    l.attended = m.out->size(1);
    l.inner = l.joint.size(1);
    pack_attention(m, l);
}

void HybridPlan::run_sandwich(const Index* ids, const b200_rows& pass, HybridCache& cache, Index max_length, void* stream, std::vector<float>* trail) {
    const Index rows = pass.rows, D = owner_.width();
    const bool planes = shadows_for(rows);
    float *h = f32(h_), *branch = f32(branch_), *projected = f32(projected_);
    const auto& runs = owner_.runs();
    float* inner_plain = planes ? nullptr : f32(plain_inner_);
    auto* inner_hi = planes ? static_cast<std::uint16_t*>(i_.hi.mutable_data()) : nullptr;
    auto* inner_lo = planes ? static_cast<std::uint16_t*>(i_.lo.mutable_data()) : nullptr;
    n_.parts = i_.parts = 0;   // the norms are finished where they are written
    // the stream's next norm, or (in front of a sublayer without a norm before it) the stream, as planes or f32 rows
    auto normed_to = [&](auto& args) {
        if (planes) { args.normed_hi = n_.hi.mutable_data(); args.normed_lo = n_.lo.mutable_data(); }
        else args.normed = f32(plain_);
    };
    if (!owner_.pairs()) {
        if (planes) {
            runtime::check(b200_embedding_shadow(owner_.embed().raw_data(), code_of(owner_.dtype()), ids, rows, owner_.vocabulary(), D,
                                                 nullptr, B200_F32, h, n_.hi.mutable_data(), n_.lo.mutable_data(), f32(squares_), stream), "embedding");
        } else {
            for (float* to : {h, f32(plain_)}) {
                runtime::check(b200_embedding_scaled(owner_.embed().raw_data(), code_of(owner_.dtype()), ids, rows, owner_.vocabulary(), D, 1.0f, to, stream), "embedding");
            }
        }
        probe(2);
    } else {
        const auto& hash = owner_.pair_hash();
        b200_pair_embedding e{};
        e.table = owner_.embed().raw_data(); e.pairs = owner_.pairs()->raw_data(); e.dtype = code_of(owner_.dtype());
        e.vocab = owner_.vocabulary(); e.width = D; e.buckets = hash.buckets; e.mul_prev = hash.mul_prev; e.mul_cur = hash.mul_cur;
        e.last = cache.last_tokens();
        e.next = layers_[static_cast<std::size_t>(runs.front().layer)].norm1.weight.data<float>(); e.eps = owner_.eps();
        e.x = h;
        normed_to(e);
        runtime::check(b200_embed_pairs(&e, ids, &pass, stream), "embedding");
        probe(2);
    }
    if (grouped_) runtime::check_cuda(cudaMemsetAsync(counts_.mutable_data(), 0, counts_.nbytes(), static_cast<cudaStream_t>(stream)), "cudaMemsetAsync");
    // the end of a sublayer whose result is in `branch`
    auto sandwich_args = [&](const Norm& after, const Norm& next) {
        b200_sandwich a{};
        a.after = after.weight.data<float>(); a.eps = owner_.eps();
        if (next.weight.defined()) a.next = next.weight.data<float>();
        else a.plain = 1;
        a.residual = h; a.x = h;
        normed_to(a);
        return a;
    };
    auto finish = [&](const Norm& after, const Norm& next) {
        const b200_sandwich a = sandwich_args(after, next);
        runtime::check(b200_sandwich_rows(branch, rows, D, &a, stream), "norms around a sublayer");
        probe(2);
    };
    auto project = [&](const void* w, Index out, float* y, const char* what) {
        if (planes) shadow(n_, rows, D, w, out, B200_EPI_STORE, nullptr, y, nullptr, nullptr, stream, what);
        else linear(f32(plain_), rows, D, w, out, B200_EPI_STORE, nullptr, y, stream, what);
    };
    auto project_inner = [&](Index inner, const void* w, const char* what) {
        if (planes) shadow(i_, rows, inner, w, D, B200_EPI_STORE, nullptr, branch, nullptr, nullptr, stream, what);
        else linear(f32(plain_inner_), rows, inner, w, D, B200_EPI_STORE, nullptr, branch, stream, what);
    };
    for (std::size_t i = 0; i < runs.size(); ++i) {
        const HybridLayer& module = *owner_.layers()[static_cast<std::size_t>(runs[i].layer)];
        const Layer& layer = layers_[static_cast<std::size_t>(runs[i].layer)];
        const Norm& next = i + 1 == runs.size() ? final_norm_ : layers_[static_cast<std::size_t>(runs[i + 1].layer)].norm1;
        // ---- mixer ----
        project(layer.in, layer.wide_out, projected, "mixer projection");
        if (module.delta) {
            run_delta(i, pass, cache, stream);
        } else {
            const b200_chunk_args a = chunk_args(layer, module, cache, i, layer.wide_out);
            runtime::check(b200_chunk_prepare(&a, &pass, nullptr, nullptr, stream), "attention norms");
            probe(2);
            runtime::check(b200_chunk_attention(&a, &pass, static_cast<int32_t>(max_length), scratch_.mutable_data(), scratch_.nbytes(), inner_plain, inner_hi, inner_lo,
                                                layer.inner, stream), "grouped attention");
            probe(1);
        }
        if (module.lightning) {
            const auto& c = module.lightning->config();
            b200_ssm_args r{};
            r.heads = r.groups = static_cast<int32_t>(c.heads); r.vdim = static_cast<int32_t>(c.vdim); r.state = static_cast<int32_t>(c.dim); r.taps = 1;
            r.ssm_state = f32(cache.run(i).state);
            r.projected = projected + layer.lightning_column; r.stride = layer.wide_out;
            r.mixed = f32(mixed_); r.y = f32(y_); r.decay = layer.decay.data<float>();
            runtime::check(b200_ssm_forward(&r, &pass, stream), "lightning recurrence");
            probe(1);
            runtime::check(b200_norm_gated(r.y, r.projected, layer.wide_out, layer.right_norm.data<float>(), rows, module.lightning->inner(), 1, owner_.eps(),
                                           static_cast<float>(module.lightning_scale), inner_plain ? inner_plain + layer.attended : nullptr,
                                           inner_hi ? inner_hi + layer.attended : nullptr, inner_lo ? inner_lo + layer.attended : nullptr, layer.inner, stream),
                           "gated norm");
            probe(2);
        }
        project_inner(layer.inner, layer.out, "output projection");
        const bool feeds = module.has_mlp() || module.mixture;
        finish(layer.after1, feeds ? layer.norm2 : next);
        // ---- feed-forward ----
        if (module.has_mlp()) {
            const Index ff = module.gate->size(0);
            if (planes) {
                shadow(n_, rows, D, layer.gate_up.raw_data(), 2 * ff, B200_EPI_SWIGLU, nullptr, nullptr, nullptr, &i_, stream, "gate/up projection", 0, 0, &layer.unit);
            } else {
                runtime::check(b200_linear_units(f32(plain_), rows, D, layer.gate_up.raw_data(), code_of(owner_.dtype()), 2 * ff, &layer.unit, f32(plain_inner_), stream),
                               "gate/up projection");
                probe(0);
            }
            project_inner(ff, layer.down, "down projection");
            finish(layer.after2, next);
        } else if (module.mixture) {
            b200_experts e = expert_args(layer, *module.mixture, rows);
            const bool sorted = b200_experts_takes_grouped(&e) != 0;
            b200_route route{};
            route.experts = static_cast<int32_t>(module.mixture->config().outputs()); route.top = e.top; route.identity = e.identity;
            route.softmax = module.mixture->config().kind.softmax;
            route.chosen_softmax = module.mixture->config().kind.chosen_softmax;
            route.bias = layer.router_bias.defined() ? layer.router_bias.data<float>() : nullptr;
            route.correction = layer.correction.defined() ? layer.correction.data<float>() : nullptr;
            route.chosen = static_cast<std::int32_t*>(chosen_.mutable_data()); route.weight = f32(score_);
            if (sorted) {
                route.rank = static_cast<std::int32_t*>(rank_.mutable_data());
                route.counts = static_cast<std::int32_t*>(counts_.mutable_data()) + static_cast<Index>(i) * (counts_.numel() / static_cast<Index>(runs.size()));
            }
            project(layer.router.raw_data(), layer.router.size(0), f32(route_logits_), "router");
            runtime::check(b200_route_rows(route_logits_.data<float>(), rows, layer.router.size(0), &route, stream), "router's choice");
            probe(2);
            e.residual = nullptr;
            if (sorted) {
                const b200_sandwich after = sandwich_args(layer.after2, next);
                e.y = nullptr;
                e.after = &after;
                runtime::check(b200_experts_grouped(&e, route.rank, route.counts, expert_scratch_.mutable_data(), expert_scratch_.nbytes(), stream), "experts");
                probe(0);
            } else {
                e.y = branch;
                runtime::check(b200_experts_streamed(&e, f32(expert_act_), stream), "experts");
                probe(0);
                finish(layer.after2, next);
            }
        }
        if (trail) keep_rows(rows, *trail);
    }
}

}  // namespace dl::nn
