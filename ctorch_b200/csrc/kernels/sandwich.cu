// Residual stream of decoders with a norm behind every sublayer (sandwich.cuh), their embedding of token pairs, and capped logits.
#include "sandwich.cuh"

#include <algorithm>

namespace b200 {
namespace {

template <int V> __global__ void __launch_bounds__(kSandwichThreads) sandwich_kernel(const float* y, const int width, const __grid_constant__ SandwichView a) {
    __shared__ float scratch[32];
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    finish_sandwich<V, true>(a, row, width, [&](int c) { return load_lanes<V>(y + row * width + c); }, scratch);
}

struct PairParams {
    const void *table, *pairs;
    int64_t vocab, buckets, mul_prev, mul_cur;
    int width;
    const int32_t* last;
    const int64_t* ids;
};

template <int V, class T> __device__ __forceinline__ Lanes<V> load_table(const T* at) {
    Lanes<V> r;
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 q = *reinterpret_cast<const uint2*>(at);
        r.v[0] = bf16_lo(q.x); r.v[1] = bf16_hi(q.x); r.v[2] = bf16_lo(q.y); r.v[3] = bf16_hi(q.y);
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) r.v[i] = load_as_f32(at, i);
    }
    return r;
}

template <class T, int V>
__global__ void __launch_bounds__(kSandwichThreads) embed_pairs_kernel(const __grid_constant__ PairParams p, const RowsView rows, const __grid_constant__ SandwichView a,
                                                                       int32_t* status) {
    __shared__ float scratch[32];
    grid_dependency_wait();   // the ids may come from the previous step's token feedback
    grid_launch_dependents();
    const int row = blockIdx.x;
    const RowPlace place = row_place(rows, row);
    int64_t id = p.ids[row];
    if (id < 0 || id >= p.vocab) {   // the host API validates ids it can see; device-resident ids are clamped and flagged
        if (threadIdx.x == 0) atomicExch(status, B200_BAD_ARGUMENT);
        id = id < 0 ? 0 : p.vocab - 1;
    }
    int64_t pair = p.buckets;
    if (place.position > 0) {
        const int64_t before = row > __ldg(rows.first + place.sequence) ? p.ids[row - 1] : p.last[place.slot];
        pair = (before * p.mul_prev + id * p.mul_cur) % p.buckets;
        if (pair < 0) pair += p.buckets;
    }
    const T *token_row = static_cast<const T*>(p.table) + id * p.width, *pair_row = static_cast<const T*>(p.pairs) + pair * p.width;
    finish_sandwich<V, false>(a, row, p.width, [&](int c) {
        Lanes<V> v = load_table<V>(token_row + c);
        const Lanes<V> w = load_table<V>(pair_row + c);
#pragma unroll
        for (int k = 0; k < V; ++k) v.v[k] += w.v[k];
        return v;
    }, scratch);
}

__global__ void soft_cap_kernel(float* x, int64_t count, float cap) {
    grid_dependency_wait();
    grid_launch_dependents();
    for (int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; i < count; i += static_cast<int64_t>(gridDim.x) * blockDim.x)
        x[i] = cap * tanhf(x[i] / cap);
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_sandwich_rows(const float* y, int64_t rows, int64_t width, const b200_sandwich* args, void* stream) {
    SandwichView a;
    if (!y || rows < 0 || width <= 0 || width > INT32_MAX || !sandwich_view(args, a)) { set_error("b200_sandwich_rows: bad pointer or size"); return B200_BAD_ARGUMENT; }
    if (rows == 0) return B200_OK;
    const bool quads = sandwich_takes_quads(a, width) && (reinterpret_cast<uintptr_t>(y) & 15) == 0;
    return cuda_status(launch_dependent(quads ? sandwich_kernel<4> : sandwich_kernel<1>, dim3(static_cast<unsigned>(rows)), dim3(kSandwichThreads), 0,
                                        as_stream(stream), y, static_cast<int>(width), a), "sandwich_kernel launch");
}

int b200_embed_pairs(const b200_pair_embedding* e, const int64_t* ids, const b200_rows* pass, void* stream) {
    RowsView rows;
    if (!rows_view(pass, rows)) return B200_BAD_ARGUMENT;
    if (!e || !ids || !e->table || !e->pairs || !e->last || !e->x || e->vocab <= 0 || e->buckets <= 0 || e->width <= 0 || e->width > INT32_MAX
        || (e->dtype != B200_F32 && e->dtype != B200_BF16) || (e->next && !e->normed && !e->normed_hi) || (e->normed_hi && !e->normed_lo)) {
        set_error("b200_embed_pairs: bad pointer or size");
        return B200_BAD_ARGUMENT;
    }
    int device = 0;
    B200_CUDA(cudaGetDevice(&device));
    int32_t* status = device_status_word(device);
    if (!status) { set_error("b200_embed_pairs: the device status word could not be allocated"); return B200_NO_DEVICE; }
    const PairParams p{e->table, e->pairs, e->vocab, e->buckets, e->mul_prev, e->mul_cur, static_cast<int>(e->width), e->last, ids};
    const SandwichView a{nullptr, e->next, static_cast<float>(e->eps), nullptr, e->x, e->normed, static_cast<__nv_bfloat16*>(e->normed_hi),
                         static_cast<__nv_bfloat16*>(e->normed_lo), false};
    const bool quads = sandwich_takes_quads(a, e->width) && ((reinterpret_cast<uintptr_t>(e->table) | reinterpret_cast<uintptr_t>(e->pairs)) & 15) == 0;
    auto kernel = e->dtype == B200_BF16 ? (quads ? embed_pairs_kernel<__nv_bfloat16, 4> : embed_pairs_kernel<__nv_bfloat16, 1>)
                                        : (quads ? embed_pairs_kernel<float, 4> : embed_pairs_kernel<float, 1>);
    return cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(rows.rows)), dim3(kSandwichThreads), 0, as_stream(stream), p, rows, a, status),
                       "embed_pairs_kernel launch");
}

int b200_soft_cap(float* x, int64_t count, float cap, void* stream) {
    if (!x || count < 0 || !(cap > 0.0f)) { set_error("b200_soft_cap: bad pointer, size or cap"); return B200_BAD_ARGUMENT; }
    if (count == 0) return B200_OK;
    const unsigned ctas = static_cast<unsigned>(std::min<int64_t>((count + 255) / 256, 8192));
    return cuda_status(launch_dependent(soft_cap_kernel, dim3(ctas), dim3(256), 0, as_stream(stream), x, count, cap), "soft_cap_kernel launch");
}

}  // extern "C"
