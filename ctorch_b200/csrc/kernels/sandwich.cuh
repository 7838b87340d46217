// Rows of the residual stream where a norm stands behind a sublayer: x = residual + rms(y) * after, then rms(x) * next for the sublayer
// that follows.  One CTA of kSandwichThreads per row; the row stays in registers between the two sums of squares.
#pragma once

#include "mma.cuh"
#include "rows.cuh"

namespace b200 {

constexpr int kSandwichThreads = 256;
constexpr int kSandwichKeep = 4;   // accesses whose values a thread keeps; what a longer row has beyond them is loaded again

struct SandwichView {
    const float *after, *next;
    float eps;
    const float* residual;
    float *x, *normed;
    __nv_bfloat16 *normed_hi, *normed_lo;
    bool plain;   // no norm follows: the planes take the stream itself
};

template <int V> __device__ __forceinline__ void store_normed(const SandwichView& a, int64_t at, const Lanes<V>& r) {
    if constexpr (V == 4) {
        if (a.normed) store_lanes<V>(a.normed + at, r);
        if (a.normed_hi) {
            uint2 hi, lo;
            pack_planes(r.v[0], r.v[1], hi.x, lo.x);
            pack_planes(r.v[2], r.v[3], hi.y, lo.y);
            *reinterpret_cast<uint2*>(a.normed_hi + at) = hi;
            *reinterpret_cast<uint2*>(a.normed_lo + at) = lo;
        }
    } else {
        store_forms(r.v[0], at, a.normed, a.normed_hi, a.normed_lo);
    }
}

// `load(c)` gives V values of the row from column c on: of y (AFTER), or of x itself.
template <int V, bool AFTER, class Load>
__device__ __forceinline__ void finish_sandwich(const SandwichView& a, int64_t row, int width, Load&& load, float* scratch) {
    constexpr int kStep = kSandwichThreads * V;
    const int64_t base = row * width;
    Lanes<V> kept[kSandwichKeep];
    auto squares_of = [](const Lanes<V>& v, float total) {
#pragma unroll
        for (int k = 0; k < V; ++k) total = fmaf(v.v[k], v.v[k], total);
        return total;
    };
    const int own = threadIdx.x * V;
#pragma unroll
    for (int i = 0; i < kSandwichKeep; ++i)
        if (own + i * kStep < width) kept[i] = load(own + i * kStep);
    float factor = 1.0f;
    if constexpr (AFTER) {
        float squares = 0.0f;
#pragma unroll
        for (int i = 0; i < kSandwichKeep; ++i)
            if (own + i * kStep < width) squares = squares_of(kept[i], squares);
        for (int c = own + kSandwichKeep * kStep; c < width; c += kStep) squares = squares_of(load(c), squares);
        factor = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(width) + a.eps);
    }
    float squares = 0.0f;
    auto to_stream = [&](int c, Lanes<V> v) {
        if constexpr (AFTER) {
            const Lanes<V> w = load_lanes<V>(a.after + c), r = load_lanes<V>(a.residual + base + c);
#pragma unroll
            for (int k = 0; k < V; ++k) v.v[k] = fmaf(v.v[k] * factor, w.v[k], r.v[k]);
        }
        store_lanes<V>(a.x + base + c, v);
        if (a.plain) store_normed<V>(a, base + c, v);
        squares = squares_of(v, squares);
        return v;
    };
#pragma unroll
    for (int i = 0; i < kSandwichKeep; ++i)
        if (own + i * kStep < width) kept[i] = to_stream(own + i * kStep, kept[i]);
    for (int c = own + kSandwichKeep * kStep; c < width; c += kStep) to_stream(c, load(c));
    if (!a.next) return;
    const float inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(width) + a.eps);
    auto finish = [&](int c, Lanes<V> v) {
        const Lanes<V> w = load_lanes<V>(a.next + c);
#pragma unroll
        for (int k = 0; k < V; ++k) v.v[k] = v.v[k] * inverse * w.v[k];
        store_normed<V>(a, base + c, v);
    };
#pragma unroll
    for (int i = 0; i < kSandwichKeep; ++i)
        if (own + i * kStep < width) finish(own + i * kStep, kept[i]);
    for (int c = own + kSandwichKeep * kStep; c < width; c += kStep) finish(c, load_lanes<V>(a.x + base + c));
}

// Host: checks and converts the C struct (false: inconsistent), and whether its rows take 16-byte accesses.
inline bool sandwich_view(const b200_sandwich* a, SandwichView& v) {
    if (!a || !a->after || !a->residual || !a->x || (a->next && !a->normed && !a->normed_hi) || (a->normed_hi && !a->normed_lo)
        || (a->plain && (a->next || (!a->normed && !a->normed_hi))))
        return false;
    v = SandwichView{a->after, a->next, static_cast<float>(a->eps), a->residual, a->x, a->normed, static_cast<__nv_bfloat16*>(a->normed_hi),
                     static_cast<__nv_bfloat16*>(a->normed_lo), a->plain != 0};
    return true;
}
inline bool sandwich_takes_quads(const SandwichView& v, int64_t width) {
    return width % 4 == 0
        && ((reinterpret_cast<uintptr_t>(v.after) | reinterpret_cast<uintptr_t>(v.next) | reinterpret_cast<uintptr_t>(v.residual) | reinterpret_cast<uintptr_t>(v.x)
             | reinterpret_cast<uintptr_t>(v.normed) | (reinterpret_cast<uintptr_t>(v.normed_hi) << 1) | (reinterpret_cast<uintptr_t>(v.normed_lo) << 1)) & 15) == 0;
}

}  // namespace b200
