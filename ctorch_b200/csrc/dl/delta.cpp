// The gated delta rule as a mixer of the configured decoders (see hybrid.h).
#include "dl/hybrid_plan.h"

#include <stdexcept>

namespace dl::nn {

DeltaMixer::DeltaMixer(Index width, const DeltaConfig& c, TensorOptions options) : config_(c) {
    if (c.heads % c.kv_heads) throw std::invalid_argument("delta rule: heads must be a multiple of kv_heads");
    if (c.dim > B200_SSM_MAX_STATE) throw std::invalid_argument("delta rule: 'dim' exceeds " + std::to_string(B200_SSM_MAX_STATE));
    auto convolved = [&](const char* name, Index rows, Tensor*& weight, Tensor*& conv) {
        weight = &register_parameter(name, host_zeros({rows, width}, options));
        conv = &register_parameter(std::string(name) + ".conv", host_zeros({rows, c.taps}, options));
    };
    convolved("q", c.kv_heads * c.dim, q, q_conv);
    convolved("k", c.kv_heads * c.dim, k, k_conv);
    convolved("v", inner(), v, v_conv);
    beta = &register_parameter("b", host_zeros({c.heads, width}, options));
    a_log = &register_parameter("A_log", host_zeros({c.heads}, options));
    norm = &register_parameter("norm", ones({c.vdim}, options));
    rate = &register_parameter("a", host_zeros({c.heads, width}, options));
    dt_bias = &register_parameter("dt_bias", host_zeros({c.heads}, options));
    gate = &register_parameter("g", host_zeros({inner(), width}, options));
    out = &register_parameter("o", host_zeros({width, inner()}, options));
}

// Rows in the order of the recurrence's columns: the gate stands where a state-space layer has its own, v, k and q in the places of x, B
// and C, the decays' inputs in that of dt.
void HybridPlan::pack_delta(const DeltaMixer& m, Layer& l) const {
    const Device where = m.q->device();
    std::vector<Tensor> rows{*m.gate, *m.v, *m.k, *m.q, *m.rate, *m.beta};
    l.wide_out = m.inner() + m.channels() + 2 * m.config().heads;
    if (const Index rest = l.wide_out % 8) {
        rows.push_back(zeros({8 - rest, owner_.width()}, {owner_.dtype(), where}));
        l.wide_out += 8 - rest;
    }
    l.wide = concat_rows(rows);
    l.in = l.wide.raw_data();
    l.out = m.out->raw_data();
    l.inner = m.inner();
    const Tensor taps[3] = {*m.v_conv, *m.k_conv, *m.q_conv};
    l.conv = to_f32(concat_rows(taps));
    l.conv_bias = zeros({m.channels()}, {DType::f32, where});
    l.dt_bias = to_f32(*m.dt_bias);
    l.a_log = to_f32(*m.a_log);
    l.gated_norm = to_f32(*m.norm);
}

void HybridPlan::run_delta(std::size_t run, const b200_rows& pass, HybridCache& cache, void* stream) {
    const auto index = static_cast<std::size_t>(owner_.runs()[run].layer);
    const Layer& layer = layers_[index];
    const auto& c = owner_.layers()[index]->delta->config();
    const bool planes = shadows_for(pass.rows);
    b200_ssm_args a{};
    a.heads = static_cast<int32_t>(c.heads); a.groups = static_cast<int32_t>(c.kv_heads); a.vdim = static_cast<int32_t>(c.vdim);
    a.state = static_cast<int32_t>(c.dim); a.taps = static_cast<int32_t>(c.taps);
    a.conv_weight = layer.conv.data<float>(); a.conv_bias = layer.conv_bias.data<float>(); a.dt_bias = layer.dt_bias.data<float>();
    a.a_log = layer.a_log.data<float>();
    a.conv_state = f32(cache.run(run).conv); a.ssm_state = f32(cache.run(run).state);
    a.projected = f32(projected_); a.stride = layer.wide_out; a.mixed = f32(mixed_); a.y = f32(y_);
    a.delta = 1;
    runtime::check(b200_ssm_forward(&a, &pass, stream), "delta rule");
    probe(1);
    runtime::check(b200_head_norm_gated(a.y, a.projected, layer.wide_out, layer.gated_norm.data<float>(), pass.rows, a.heads, a.vdim, owner_.eps(),
                                        planes ? nullptr : f32(plain_inner_), planes ? i_.hi.mutable_data() : nullptr, planes ? i_.lo.mutable_data() : nullptr,
                                        layer.inner, stream), "gated norm");
    probe(2);
}

}  // namespace dl::nn
