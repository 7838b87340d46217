// Device view of a packed pass (b200_rows): which sequence, cache slot and position every activation row has.
#pragma once

#include "common.cuh"

namespace b200 {

struct RowsView {
    int rows, sequences, max_count;
    const int32_t *slot, *first, *sequence;
    int32_t* lengths;
};

struct RowPlace { int sequence, slot, position; };

__device__ __forceinline__ RowPlace row_place(const RowsView& v, int row) {
    const int s = __ldg(v.sequence + row), slot = __ldg(v.slot + s);
    return {s, slot, v.lengths[slot] + row - __ldg(v.first + s)};
}

// Checks and converts the C struct; false (with the error text set) when it is inconsistent.
bool rows_view(const b200_rows* pass, RowsView& view);

// Two bf16 planes of an f32 value (hi + lo, about 16 mantissa bits).
__device__ __forceinline__ void split_planes(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(v);
    lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
// One result of a row kernel to whichever forms are wanted.
__device__ __forceinline__ void store_forms(float v, int64_t at, float* out, __nv_bfloat16* out_hi, __nv_bfloat16* out_lo) {
    if (out) out[at] = v;
    if (out_hi) {
        __nv_bfloat16 hi, lo;
        split_planes(v, hi, lo);
        out_hi[at] = hi;
        if (out_lo) out_lo[at] = lo;
    }
}

// V adjacent f32 values, 4 on a 16-byte boundary or 1.
template <int V> struct Lanes { float v[V]; };
template <int V> __device__ __forceinline__ Lanes<V> load_lanes(const float* p) {
    Lanes<V> r;
    if constexpr (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    } else {
        r.v[0] = p[0];
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_lanes(float* p, const Lanes<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else p[0] = r.v[0];
}

// Sum over the CTA (any block size that is a multiple of 32, at most 1024); every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    const int warps = blockDim.x >> 5;
    float total = 0.0f;
    for (int w = 0; w < warps; ++w) total += scratch[w];
    return total;
}

}  // namespace b200
