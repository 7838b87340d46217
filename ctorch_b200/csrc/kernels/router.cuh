// Choice of a router: the outputs with the largest scores, by one warp per row (b200_route).
#pragma once

#include "common.cuh"

namespace b200 {

struct Route {
    int experts, top;
    int64_t column;
    int32_t* chosen;
    float* weight;
    int32_t *rank, *counts;
    bool softmax;
    const float* correction;
    int identity;
    const float* bias;
    bool chosen_softmax;
};

// Checks and converts the C struct; false when it is inconsistent.
inline bool route_view(const b200_route* r, Route& view) {
    if (r->experts <= 0 || r->experts > B200_MAX_EXPERTS || r->top <= 0 || r->top > r->experts || r->column < 0 || !r->chosen || !r->weight
        || (r->rank && !r->counts) || (r->chosen_softmax && (r->softmax || r->correction)) || r->identity < 0 || r->identity > r->experts)
        return false;
    view = Route{r->experts, r->top, r->column, r->chosen, r->weight, r->rank, r->counts, r->softmax != 0, r->correction, r->identity, r->bias,
                 r->chosen_softmax != 0};
    return true;
}

// The `top` outputs with the largest choice scores, the lower index among equals, and their weights.  `copy` [experts] is shared memory of
// this warp.  Sigmoid scores grow with the logits, which are therefore compared themselves while nothing is added to the scores.
__device__ __forceinline__ void choose_experts(const Route& r, int row, const float* logits, float* copy, int lane) {
    const bool scored = r.softmax || r.correction;
    float high = 0.0f, inverse = 1.0f;
    auto logit = [&](int e) { return r.bias ? logits[e] + __ldg(r.bias + e) : logits[e]; };
    if (r.softmax) {
        high = -INFINITY;
        for (int e = lane; e < r.experts; e += 32) high = fmaxf(high, logit(e));
        high = warp_max(high);
        float total = 0.0f;
        for (int e = lane; e < r.experts; e += 32) total += expf(logit(e) - high);
        inverse = 1.0f / warp_sum(total);
    }
    auto score = [&](int e) { return r.softmax ? expf(logit(e) - high) * inverse : 1.0f / (1.0f + expf(-logit(e))); };
    for (int e = lane; e < r.experts; e += 32) copy[e] = scored ? score(e) + (r.correction ? r.correction[e] : 0.0f) : logit(e);
    __syncwarp();
    for (int k = 0; k < r.top; ++k) {
        float best = -INFINITY;
        int at = INT32_MAX;
        for (int e = lane; e < r.experts; e += 32)
            if (copy[e] > best || at == INT32_MAX) { best = copy[e]; at = e; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float other = __shfl_xor_sync(0xffffffffu, best, o);
            const int other_at = __shfl_xor_sync(0xffffffffu, at, o);
            if (other_at != INT32_MAX && (at == INT32_MAX || other > best || (other == best && other_at < at))) { best = other; at = other_at; }
        }
        if (lane == 0) {
            const int64_t slot = static_cast<int64_t>(row) * r.top + k;
            r.chosen[slot] = at;
            if (r.chosen_softmax) {
                if (k == 0) high = logit(at);
                r.weight[slot] = expf(logit(at) - high);   // divided by their sum below
            } else {
                r.weight[slot] = score(at);
            }
            if (r.rank && at < r.experts - r.identity) r.rank[slot] = atomicAdd(r.counts + at, 1);
            copy[at] = -INFINITY;
        }
        __syncwarp();
    }
    if (!r.chosen_softmax) return;
    float* weight = r.weight + static_cast<int64_t>(row) * r.top;
    float total = 0.0f;
    for (int k = lane; k < r.top; k += 32) total += weight[k];
    total = warp_sum(total);
    for (int k = lane; k < r.top; k += 32) weight[k] /= total;
}

}  // namespace b200
