// Grouped-query attention over slots.  With chunks a position sees its own chunk of positions up to itself, so a slot keeps one chunk of
// keys and values ([slot][kv_head][entry][dim], position p in entry p mod chunk) however long the sequence grows; without chunks it keeps
// all of them.  What a step reads is one contiguous block per (sequence, kv head).  Keys and values may have different widths.
//
//   * chunk_prepare_kernel, one CTA per row (and one per slice of its feed-forward units): biases, RMS norms (over all heads at once or per
//     head), rotation of halves or of adjacent pairs, append (or the workspaces of a longer pass), the activation of feed-forward units and
//     the router's choice for the same row.
//   * chunk_step_kernel, chunk_mma_kernel: bf16, mma.sync products, online softmax in f32 registers, weights as hi + lo planes, the heads
//     of a group side by side so that a key is fetched once for all of them.  Scores may be capped (softcap * tanh), and the denominator
//     may hold a term without a key (sink), which joins the sums when a row is finished.
//       steps (one row per sequence): bound by the keys' bytes.  Persistent CTAs walk (sequence, kv head, split) items; a producer warp
//         streams tiles of 64 keys and values through a TMA ring (boxes of 64 x 64, 128-byte swizzle, mbarrier completion) and runs
//         into the next item while four consumer warps, which divide the keys of a tile, merge the current one.  Keys are split over
//         CTAs, with a merge kernel, where the items do not fill the SMs;
//       longer passes: 64 rows = positions x heads of a group, 16 per warp, a cp.async double buffer; keys before the pass come from the
//         slot, the pass's own keys from its workspaces (from the slot too without chunks, where they are appended first).
//   * chunk_generic_kernel: f32 and odd sizes, f32 FMAs, one (row, head) per CTA.
//   * chunk_append_kernel: a longer pass that begins inside a chunk and ends in another one reads the old chunk from the slot; its last
//     rows go there afterwards.
#include "mma.cuh"
#include "router.cuh"
#include "rows.cuh"

#include <algorithm>
#include <type_traits>

namespace b200 {
namespace {

struct ChunkParams {
    int heads, kv_heads, group, dim, vdim, rot_dims, slots, chunk, entries;
    float scale, eps;
    const float *cosine, *sine;
    int positions;
    const float *q_norm, *k_norm;
    void *key_cache, *value_cache, *query, *key, *value;
    const float* projected;
    int64_t stride;
    const float *q_bias, *k_bias, *sink;
    int norm;
    bool rotate_pairs, keys_as_values, keys_elsewhere, gated;
    float softcap, out_scale;
    int window, keep, pool;
    float* pool_state;
    bool norm_values, gate_values;
    const float* talk;
    size_t table_bytes;
    __host__ __device__ __forceinline__ int key_columns() const { return keys_elsewhere ? 0 : kv_heads * dim; }
    __host__ __device__ __forceinline__ int value_columns() const { return keys_elsewhere || keys_as_values ? 0 : kv_heads * vdim; }
    // Keys of the pass itself are in the slots before the attention starts.
    __host__ __device__ __forceinline__ bool appends_first(bool step) const { return step || (chunk == 0 && window == 0); }
    __device__ __forceinline__ int chunk_start(int position) const { return chunk > 0 ? position - position % chunk : 0; }
    // The entry that holds a position: of its chunk, of the first positions that stay, or of the window's ring.
    __device__ __forceinline__ int place(int position) const {
        if (window > 0) return position < keep ? position : keep + (position - keep) % window;
        return position - chunk_start(position);
    }
    // where (slot, kv head)'s entry number `place` begins, in units of one entry
    __device__ __forceinline__ int64_t entry_at(int slot, int head, int at) const { return (static_cast<int64_t>(slot) * kv_heads + head) * entries + at; }
    __device__ __forceinline__ int64_t entry(int slot, int head, int position) const { return entry_at(slot, head, place(position)); }
    // The first position of the run of positions up to itself that `position` sees; and, before it, the kept positions or pooled blocks.
    __device__ __forceinline__ int first_seen(int position) const { return window > 0 ? max(0, position - window + 1) : chunk_start(position); }
    __device__ __forceinline__ int blocks_seen(int position) const { return position < window ? 0 : (position - window + 1) / pool; }
    __device__ __forceinline__ int before_run(int position) const { return pool > 0 ? blocks_seen(position) : min(keep, first_seen(position)); }
    // Entries that a position sees once it is in its slot: they are the first ones of the slot, in whatever order.
    __device__ __forceinline__ int entries_seen(int position) const {
        if (window > 0) return min(position + 1, keep + window) + (pool > 0 ? blocks_seen(position) : 0);
        return position - chunk_start(position) + 1;
    }
    // Whether storing the rows of a pass from position `length` to `last` overwrites keys that the pass itself still reads.
    __device__ __forceinline__ bool overwrites(int length, int last) const {
        return window > 0 ? length > 0 : chunk > 0 && length % chunk != 0 && chunk_start(length) != chunk_start(last);
    }
    // Whether a position's key is still of use behind position `last`.
    __device__ __forceinline__ bool outlasts(int position, int last) const {
        return window > 0 ? position < keep || position > last - window : chunk_start(position) == chunk_start(last);
    }
    __device__ __forceinline__ bool fits(int position) const { return place(position) < entries; }
};
// Head dimensions from which lanes are handed out to a head: a power of two of neighbouring lanes, as many as its values occupy.
__device__ __forceinline__ int lanes_per_head(int size, int per_lane) { return size > 16 * per_lane ? 32 : size > 8 * per_lane ? 16 : 8; }

bool chunk_params(const b200_chunk_args* a, ChunkParams& p) {
    if (!a || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->rot_dims < 0 || (a->rot_dims & 1)
        || a->rot_dims > a->dim || a->slots <= 0 || a->chunk < 0 || a->entries <= 0 || (a->rot_dims > 0 && (!a->cosine || !a->sine))
        || (a->norm == B200_HEAD_NORM_PROJECTION && (!a->q_norm || (!a->k_norm && !a->keys_elsewhere)))
        || a->norm < B200_HEAD_NORM_PROJECTION || a->norm > B200_HEAD_NORM_HEAD || (a->keys_elsewhere && a->chunk > 0)
        || (a->keys_as_values && (a->vdim != a->dim || a->norm != B200_HEAD_NORM_NONE)) || !(a->softcap >= 0.0f)
        || a->window < 0 || a->keep < 0 || a->pool < 0 || (a->window > 0 && (a->chunk > 0 || a->keys_elsewhere || a->entries < a->keep + a->window))
        || ((a->keep > 0 || a->pool > 0) && a->window == 0) || (a->pool > 0 && (a->keep > 0 || !a->pool_state)) || (a->talk && a->sink)
        || (a->norm == B200_HEAD_NORM_HEAD && !a->q_norm != !a->k_norm && !a->keys_elsewhere) || (a->gate_values && !a->no_gate)
        || (a->dtype != B200_F32 && a->dtype != B200_BF16) || !a->key_cache || !a->value_cache || !a->projected || !a->query || a->stride <= 0) {
        set_error("grouped attention: bad pointer or size");
        return false;
    }
    p = ChunkParams{a->heads, a->kv_heads, a->heads / a->kv_heads, a->dim, a->vdim, a->rot_dims, a->slots, a->chunk, a->entries, a->scale, static_cast<float>(a->eps),
                    a->cosine, a->sine, a->positions, a->q_norm, a->k_norm, a->key_cache, a->value_cache, a->query, a->key, a->value, a->projected, a->stride,
                    a->q_bias, a->k_bias, a->sink, a->norm, a->rotate_pairs != 0, a->keys_as_values != 0, a->keys_elsewhere != 0, a->no_gate == 0, a->softcap,
                    a->scaled ? a->out_scale : 1.0f, a->window, a->keep, a->pool, a->pool_state, a->norm_values != 0, a->gate_values != 0, a->talk, static_cast<size_t>(std::max<int64_t>(0, a->table_bytes))};
    if (p.heads * p.dim + p.key_columns() + p.value_columns() + (p.gate_values ? p.heads * p.vdim : p.gated ? p.heads : 0) > p.stride) {
        set_error("grouped attention: the projected rows are shorter than the heads");
        return false;
    }
    return true;
}

// ---- between the projection and the attention -----------------------------------------------------------------------
struct Units { int kind; int64_t column; int count; float* out; __nv_bfloat16 *out_hi, *out_lo; int64_t stride; };

template <int V> struct Span { float v[V]; };
template <int V> __device__ __forceinline__ Span<V> load_span(const float* p) {
    Span<V> r;
    if constexpr (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_span(float* p, const Span<V>& s) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(s.v[0], s.v[1], s.v[2], s.v[3]);
    else *p = s.v[0];
}
template <int V> __device__ __forceinline__ void store_span(__nv_bfloat16* p, const Span<V>& s) {
    if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(s.v[0], s.v[1]), pack_bf16(s.v[2], s.v[3]));
    else *p = __float2bfloat16_rn(s.v[0]);
}
// The value that a cache of T holds for v.
template <class T> __device__ __forceinline__ float rounded_to(float v) {
    if constexpr (sizeof(T) == 2) return __bfloat162float(__float2bfloat16_rn(v));
    else return v;
}
// Entries [c, c + V) of a projected row's part, with its bias.
template <int V> __device__ __forceinline__ Span<V> biased_span(const float* x, const float* bias, int c) {
    Span<V> s = load_span<V>(x + c);
    if (bias) {
        const Span<V> b = load_span<V>(bias + c);
#pragma unroll
        for (int i = 0; i < V; ++i) s.v[i] += b.v[i];
    }
    return s;
}
// This thread's share of the sum of squares of entries [begin, end), `threads` threads side by side.
template <int V> __device__ __forceinline__ float squares_of(const float* x, const float* bias, int begin, int end, int thread, int threads) {
    float total = 0.0f;
    for (int c = begin + thread * V; c < end; c += threads * V) {
        const Span<V> s = biased_span<V>(x, bias, c);
#pragma unroll
        for (int i = 0; i < V; ++i) total = fmaf(s.v[i], s.v[i], total);
    }
    return total;
}
// V entries from entry c of a part on, which is entry d of its head: with bias, normed, weighted (weight may be NULL; PER_HEAD: the same for
// every head), and turned by the row's angles - entry i with entry i + rot_dims / 2, or entry 2i with entry 2i + 1.
template <int V, bool PER_HEAD = false>
__device__ __forceinline__ Span<V> turned_span(const ChunkParams& p, const float* part, const float* bias, const float* weight, int c, int d, float inverse,
                                               const float* cosine, const float* sine) {
    auto normed = [&](int at) {
        Span<V> s = biased_span<V>(part, bias, at);
        if (weight) {
            const Span<V> w = load_span<V>(weight + (PER_HEAD ? at - c + d : at));
#pragma unroll
            for (int i = 0; i < V; ++i) s.v[i] = s.v[i] * inverse * w.v[i];
        } else {
#pragma unroll
            for (int i = 0; i < V; ++i) s.v[i] *= inverse;
        }
        return s;
    };
    Span<V> own = normed(c);
    if (d >= p.rot_dims || !cosine) return own;
    if (p.rotate_pairs) {
        if constexpr (V == 1) {
            const float other = normed(d & 1 ? c - 1 : c + 1).v[0], cs = cosine[d >> 1], sn = sine[d >> 1];
            own.v[0] = d & 1 ? __fadd_rn(__fmul_rn(own.v[0], cs), __fmul_rn(other, sn)) : __fsub_rn(__fmul_rn(own.v[0], cs), __fmul_rn(other, sn));
        } else {
#pragma unroll
            for (int i = 0; i < V; i += 2) {
                if (d + i >= p.rot_dims) break;
                const float cs = cosine[(d + i) >> 1], sn = sine[(d + i) >> 1], u = own.v[i], v = own.v[i + 1];
                own.v[i] = __fsub_rn(__fmul_rn(u, cs), __fmul_rn(v, sn));
                own.v[i + 1] = __fadd_rn(__fmul_rn(v, cs), __fmul_rn(u, sn));
            }
        }
        return own;
    }
    const int half = p.rot_dims >> 1;
    const bool upper = d >= half;
    const Span<V> other = normed(upper ? c - half : c + half);
    const Span<V> cs = load_span<V>(cosine + (upper ? d - half : d)), sn = load_span<V>(sine + (upper ? d - half : d));
#pragma unroll
    for (int i = 0; i < V; ++i)
        own.v[i] = upper ? __fadd_rn(__fmul_rn(own.v[i], cs.v[i]), __fmul_rn(other.v[i], sn.v[i]))
                         : __fsub_rn(__fmul_rn(own.v[i], cs.v[i]), __fmul_rn(other.v[i], sn.v[i]));
    return own;
}

constexpr int kPrepareThreads = 256, kUnitSlice = 1024;
// grid (rows, 1 + slices of the units)

// NORM: b200_head_norm
template <class T, int V, int NORM>
__global__ void __launch_bounds__(kPrepareThreads) chunk_prepare_kernel(const __grid_constant__ ChunkParams p, const RowsView rows, const bool step,
                                                                        const __grid_constant__ Units units, const __grid_constant__ Route route) {
    extern __shared__ float logits_copy[];
    __shared__ float scratch[32];
    grid_dependency_wait();
    grid_launch_dependents();
    const int row = blockIdx.x;
    const float* source = p.projected + row * p.stride;
    if (blockIdx.y > 0) {   // a slice of the row's feed-forward units
        const float* from = source + units.column;
        const int begin = (blockIdx.y - 1) * kUnitSlice, end = min(units.count, begin + kUnitSlice);
        auto store = [&](int j, const Span<V>& v) {
            const int64_t at = row * units.stride + j;
            if (units.out) store_span<V>(units.out + at, v);
            if (units.out_hi) {
                Span<V> rest;
#pragma unroll
                for (int i = 0; i < V; ++i) rest.v[i] = v.v[i] - __bfloat162float(__float2bfloat16_rn(v.v[i]));
                store_span<V>(units.out_hi + at, v);
                store_span<V>(units.out_lo + at, rest);
            }
        };
        for (int j = begin + threadIdx.x * V; j < end; j += kPrepareThreads * V) {
            Span<V> v;
            if (units.kind == 1) {
                float pairs[2 * V];
#pragma unroll
                for (int i = 0; i < 2 * V; i += V) {
                    const Span<V> part = load_span<V>(from + 2 * j + i);
#pragma unroll
                    for (int e = 0; e < V; ++e) pairs[i + e] = part.v[e];
                }
#pragma unroll
                for (int i = 0; i < V; ++i) v.v[i] = silu_reference(pairs[2 * i]) * pairs[2 * i + 1];
            } else {
                v = load_span<V>(from + j);
#pragma unroll
                for (int i = 0; i < V; ++i) v.v[i] = gelu_exact(v.v[i]);
            }
            store(j, v);
        }
        return;
    }
    if (route.experts > 0 && threadIdx.x >= kPrepareThreads - 32)
        choose_experts(route, row, source + route.column, logits_copy, threadIdx.x & 31);
    const int sequence = __ldg(rows.sequence + row);
    const int q_count = p.heads * p.dim, k_count = p.key_columns(), v_count = p.keys_elsewhere ? 0 : p.kv_heads * p.vdim;
    const float *k_source = source + q_count, *v_source = p.keys_as_values ? k_source : k_source + k_count;
    const float* v_bias = p.keys_as_values ? p.k_bias : nullptr;
    float q_inverse = 1.0f, k_inverse = 1.0f, qs = 0.0f, ks = 0.0f;
    if constexpr (NORM == B200_HEAD_NORM_PROJECTION) {
        qs = squares_of<V>(source, p.q_bias, 0, q_count, threadIdx.x, kPrepareThreads);
        ks = squares_of<V>(k_source, p.k_bias, 0, k_count, threadIdx.x, kPrepareThreads);
    }
    // where the row belongs: a chain of dependent loads, spread between the sums
    const int slot = __ldg(rows.slot + sequence), first = __ldg(rows.first + sequence), end = __ldg(rows.first + sequence + 1);
    if constexpr (NORM == B200_HEAD_NORM_PROJECTION) {
        qs = warp_sum(qs);
        ks = warp_sum(ks);
    }
    const int length = rows.lengths[slot];
    if constexpr (NORM == B200_HEAD_NORM_PROJECTION) {
        if ((threadIdx.x & 31) == 0) { scratch[threadIdx.x >> 5] = qs; scratch[kPrepareThreads / 32 + (threadIdx.x >> 5)] = ks; }
        __syncthreads();
        qs = ks = 0.0f;
#pragma unroll
        for (int w = 0; w < kPrepareThreads / 32; ++w) { qs += scratch[w]; ks += scratch[kPrepareThreads / 32 + w]; }
        q_inverse = 1.0f / sqrtf(qs / static_cast<float>(q_count) + p.eps);
        k_inverse = 1.0f / sqrtf(ks / static_cast<float>(max(k_count, 1)) + p.eps);
    }
    const int position = length + row - first, last = length + end - first - 1;
    // The slot takes the row at once where it ends up there and nothing that this pass still reads is overwritten.
    const bool first_appended = p.appends_first(step);
    const bool stored = first_appended || (p.outlasts(position, last) && !p.overwrites(length, last));
    const bool to_slot = stored && p.fits(position);   // (the host refuses passes that do not fit)
    const int half = p.rot_dims >> 1;
    const bool turns = half > 0 && position < p.positions;
    const float* cosine = turns ? p.cosine + static_cast<int64_t>(position) * half : nullptr;
    const float* sine = turns ? p.sine + static_cast<int64_t>(position) * half : nullptr;
    auto store_query = [&](int c, const Span<V>& v) { store_span<V>(static_cast<T*>(p.query) + static_cast<int64_t>(row) * q_count + c, v); };
    // A step's share of the block that is being pooled: the sum of what the cache holds, and its mean once the block is complete.
    const int place = p.place(position);
    const bool pools = step && p.pool > 0, pool_begins = pools && position % p.pool == 0, pool_ends = pools && (position + 1) % p.pool == 0;
    auto pool_up = [&](T* cache, int size, int head, int offset, int d, const Span<V>& v) {
        float* sum = p.pool_state + (static_cast<int64_t>(slot) * p.kv_heads + head) * (p.dim + p.vdim) + offset + d;
        Span<V> total = pool_begins ? Span<V>{} : load_span<V>(sum);
#pragma unroll
        for (int i = 0; i < V; ++i) total.v[i] += rounded_to<T>(v.v[i]);
        if (!pool_ends) return store_span<V>(sum, total);
#pragma unroll
        for (int i = 0; i < V; ++i) total.v[i] /= static_cast<float>(p.pool);
        const int at = p.window + position / p.pool;
        if (at < p.entries) store_span<V>(cache + p.entry_at(slot, head, at) * size + d, total);
    };
    auto store_key = [&](int head, int d, const Span<V>& v) {
        if (to_slot) store_span<V>(static_cast<T*>(p.key_cache) + p.entry_at(slot, head, place) * p.dim + d, v);
        if (!first_appended) store_span<V>(static_cast<T*>(p.key) + static_cast<int64_t>(row) * k_count + head * p.dim + d, v);
        if (pools) pool_up(static_cast<T*>(p.key_cache), p.dim, head, 0, d, v);
    };
    auto store_value = [&](int head, int d, const Span<V>& v) {
        if (to_slot) store_span<V>(static_cast<T*>(p.value_cache) + p.entry_at(slot, head, place) * p.vdim + d, v);
        if (!first_appended) store_span<V>(static_cast<T*>(p.value) + static_cast<int64_t>(row) * v_count + head * p.vdim + d, v);
        if (pools) pool_up(static_cast<T*>(p.value_cache), p.vdim, head, p.dim, d, v);
    };
    if constexpr (NORM == B200_HEAD_NORM_HEAD) {
        // the key heads follow the query heads
        const int lanes = lanes_per_head(p.dim, V), lane = threadIdx.x & (lanes - 1), at_once = kPrepareThreads / lanes;
        const int heads = p.heads + (p.keys_elsewhere ? 0 : p.kv_heads);
        for (int h0 = 0; h0 < heads; h0 += at_once) {
            const int h = h0 + static_cast<int>(threadIdx.x) / lanes;
            const bool live = h < heads, is_query = h < p.heads;
            const float *part = is_query ? source : k_source, *bias = is_query ? p.q_bias : p.k_bias;
            const int head = is_query ? h : h - p.heads, begin = head * p.dim;
            float squares = live ? squares_of<V>(part, bias, begin, begin + p.dim, lane, lanes) : 0.0f;
            for (int o = lanes >> 1; o > 0; o >>= 1) squares += __shfl_xor_sync(0xffffffffu, squares, o);
            const float inverse = 1.0f / sqrtf(squares / static_cast<float>(p.dim) + p.eps);
            for (int d = lane * V; live && d < p.dim; d += lanes * V) {
                const Span<V> v = turned_span<V, true>(p, part, bias, is_query ? p.q_norm : p.k_norm, begin + d, d, inverse, cosine, sine);
                if (is_query) store_query(begin + d, v);
                else store_key(head, d, v);
            }
        }
    } else {
        constexpr bool kWeighted = NORM == B200_HEAD_NORM_PROJECTION;
        for (int c = threadIdx.x * V; c < q_count; c += kPrepareThreads * V)
            store_query(c, turned_span<V>(p, source, p.q_bias, kWeighted ? p.q_norm : nullptr, c, c % p.dim, q_inverse, cosine, sine));
        for (int c = threadIdx.x * V; c < k_count; c += kPrepareThreads * V) {
            const int head = c / p.dim, d = c - head * p.dim;
            store_key(head, d, turned_span<V>(p, k_source, p.k_bias, kWeighted ? p.k_norm : nullptr, c, d, k_inverse, cosine, sine));
        }
    }
    if (p.norm_values && v_count > 0) {
        const int lanes = lanes_per_head(p.vdim, V), lane = threadIdx.x & (lanes - 1), at_once = kPrepareThreads / lanes;
        for (int h0 = 0; h0 < p.kv_heads; h0 += at_once) {
            const int head = h0 + static_cast<int>(threadIdx.x) / lanes, begin = head * p.vdim;
            const bool live = head < p.kv_heads;
            float squares = live ? squares_of<V>(v_source, v_bias, begin, begin + p.vdim, lane, lanes) : 0.0f;
            for (int o = lanes >> 1; o > 0; o >>= 1) squares += __shfl_xor_sync(0xffffffffu, squares, o);
            const float inverse = 1.0f / sqrtf(squares / static_cast<float>(p.vdim) + p.eps);
            for (int d = lane * V; live && d < p.vdim; d += lanes * V) {
                Span<V> v = biased_span<V>(v_source, v_bias, begin + d);
#pragma unroll
                for (int i = 0; i < V; ++i) v.v[i] *= inverse;
                store_value(head, d, v);
            }
        }
        return;
    }
    for (int c = threadIdx.x * V; c < v_count; c += kPrepareThreads * V) {
        const int head = c / p.vdim;
        store_value(head, c - head * p.vdim, biased_span<V>(v_source, v_bias, c));
    }
}

// Before the attention of a longer pass: the blocks of `pool` positions that the pass completes, and the sum of the one it leaves open.  grid
// (blocks of a sequence, sequences, column blocks), V columns per thread; CTA 0 takes the first block, which earlier passes may have begun,
// and the open one.
constexpr int kPoolThreads = 128;
template <class T, int V> __global__ void __launch_bounds__(kPoolThreads) chunk_pool_kernel(const __grid_constant__ ChunkParams p, const RowsView rows) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int per_head = p.dim + p.vdim, c = (blockIdx.z * kPoolThreads + threadIdx.x) * V;
    if (c >= p.kv_heads * per_head) return;
    const int sequence = blockIdx.y, first = __ldg(rows.first + sequence), count = __ldg(rows.first + sequence + 1) - first;
    const int slot = __ldg(rows.slot + sequence), length = rows.lengths[slot], end = length + count;
    const int block0 = length / p.pool, block1 = (end - 1) / p.pool, head = c / per_head, d = c - head * per_head;
    const bool is_key = d < p.dim;
    const int size = is_key ? p.dim : p.vdim, at_head = is_key ? d : d - p.dim;
    const T* source = static_cast<const T*>(is_key ? p.key : p.value) + head * size + at_head;
    const int64_t stride = static_cast<int64_t>(p.kv_heads) * size;
    T* cache = static_cast<T*>(is_key ? p.key_cache : p.value_cache);
    float* sum = p.pool_state + static_cast<int64_t>(slot) * p.kv_heads * per_head + c;
    auto pool_block = [&](int block) {
        const int from = max(block * p.pool, length), to = min((block + 1) * p.pool, end), at = p.window + block;
        Span<V> total{};
        if (from > block * p.pool) total = load_span<V>(sum);
#pragma unroll 8
        for (int j = from; j < to; ++j) {
            const T* row = source + (first + j - length) * stride;
            if constexpr (V == 4 && sizeof(T) == 2) {
                const uint2 q = __ldcg(reinterpret_cast<const uint2*>(row));
                total.v[0] += bf16_lo(q.x); total.v[1] += bf16_hi(q.x); total.v[2] += bf16_lo(q.y); total.v[3] += bf16_hi(q.y);
            } else {
#pragma unroll
                for (int i = 0; i < V; ++i) total.v[i] += load_as_f32(row, i);
            }
        }
        if (to < (block + 1) * p.pool) return store_span<V>(sum, total);
#pragma unroll
        for (int i = 0; i < V; ++i) total.v[i] /= static_cast<float>(p.pool);
        if (at < p.entries) store_span<V>(cache + p.entry_at(slot, head, at) * size + at_head, total);
    };
    const int block = block0 + static_cast<int>(blockIdx.x);
    if (blockIdx.x == 0) {
        pool_block(block0);
        if (block1 > block0) pool_block(block1);   // (the same thread has read what earlier passes left)
    } else if (block < block1) {
        pool_block(block);
    }
}

// After a longer pass: the rows that later ones see (of a sequence's last chunk or window) go into its slot, where they could not before
// (see chunk_prepare_kernel).
template <class T> __global__ void __launch_bounds__(128) chunk_append_kernel(const __grid_constant__ ChunkParams p, const RowsView rows) {
    grid_dependency_wait();
    grid_launch_dependents();
    for (int row = blockIdx.x; row < rows.rows; row += gridDim.x) {
        const RowPlace place = row_place(rows, row);
        const int length = rows.lengths[place.slot];
        const int last = length + __ldg(rows.first + place.sequence + 1) - __ldg(rows.first + place.sequence) - 1;
        if (!p.overwrites(length, last) || !p.outlasts(place.position, last) || !p.fits(place.position)) continue;
        const int k_count = p.kv_heads * p.dim, v_count = p.kv_heads * p.vdim;
        for (int c = threadIdx.x; c < k_count; c += blockDim.x)
            static_cast<T*>(p.key_cache)[p.entry(place.slot, c / p.dim, place.position) * p.dim + c % p.dim] =
                static_cast<const T*>(p.key)[static_cast<int64_t>(row) * k_count + c];
        for (int c = threadIdx.x; c < v_count; c += blockDim.x)
            static_cast<T*>(p.value_cache)[p.entry(place.slot, c / p.vdim, place.position) * p.vdim + c % p.vdim] =
                static_cast<const T*>(p.value)[static_cast<int64_t>(row) * v_count + c];
    }
}

// ---- attention ------------------------------------------------------------------------------------------------------
struct ChunkAttention {
    ChunkParams p;
    RowsView rows;
    bool step;                      // one row per sequence: every key, the row's own included, is in the slots
    int stages;
    int32_t* status;
    int positions_per_tile, heads_per_tile, head_tiles, splits;
    float *partial, *partial_ml;    // splits > 1: [rows, heads, splits, vdim], [rows, heads, splits, 2]
    // mixed heads: the tables between the kernels of b200_chunk_attention, for the positions [begin, begin + span) of the sequences from
    // first_sequence on
    float *table, *table_ml;        // [sequence, position, heads, pitch] scores, then packed weights; [..., heads, splits, 2] their largest and sum
    int64_t pitch;
    int first_sequence, begin, span;
    float* out;
    __nv_bfloat16 *out_hi, *out_lo;
    int64_t out_stride;
};

// Factor of a head's result: its gate, and the layer's scale.
__device__ __forceinline__ float head_gate(const ChunkParams& p, int row, int head) {
    if (!p.gated) return p.out_scale;
    const float g = __ldg(p.projected + row * p.stride + p.heads * p.dim + p.key_columns() + p.value_columns() + head);
    return p.out_scale / (1.0f + expf(-g));
}
// A value's own gate, where every value of a head has one.
__device__ __forceinline__ float value_gate(const ChunkParams& p, int row, int head, int column) {
    const float g = __ldg(p.projected + row * p.stride + p.heads * p.dim + p.key_columns() + p.value_columns() + head * p.vdim + column);
    return 1.0f / (1.0f + expf(-g));
}
// The scores are kept in units of log2: `scale2` times the product, or cap2 * tanh(product * scale / softcap).  The tensor-core kernels take
// the hardware's exponential and reciprocal (an error near 1e-6 of the cap), the plain one the exact functions.
__device__ __forceinline__ float capped_score(float product, float scale_by_cap, float cap2) {
    const float e = exp2_fast(2.0f * kLog2e * product * scale_by_cap);   // (infinite for large scores: then the cap itself)
    return cap2 - __fdividef(2.0f * cap2, e + 1.0f);
}
// What multiplies a finished accumulator (largest score `top`, in units of log2, and sum `total` of the weights under it): the reciprocal of
// the denominator, a sink included.
__device__ __forceinline__ float denominator_factor(const ChunkParams& p, int head, float top, float total) {
    if (!p.sink) return 1.0f / total;
    const float sink = __ldg(p.sink + head) * kLog2e, high = fmaxf(top, sink);
    const float factor = exp2f(top - high);
    return factor / fmaf(total, factor, exp2f(sink - high));
}

__device__ __forceinline__ void store_pair(const ChunkAttention& a, int row, int head, int column, float x, float y) {
    const int64_t at = row * a.out_stride + head * a.p.vdim + column;
    if (a.p.gate_values) {   // (hardware exponential and division: an error near 1e-6, as in the weights)
        const ChunkParams& p = a.p;
        const float2 g = __ldg(reinterpret_cast<const float2*>(p.projected + row * p.stride + p.heads * p.dim + p.key_columns() + p.value_columns() + head * p.vdim + column));
        x = __fdividef(x, 1.0f + exp2_fast(-kLog2e * g.x));
        y = __fdividef(y, 1.0f + exp2_fast(-kLog2e * g.y));
    }
    if (a.out) *reinterpret_cast<float2*>(a.out + at) = make_float2(x, y);
    if (a.out_hi) {
        uint32_t hi, lo;
        pack_planes(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(a.out_hi + at) = hi;
        if (a.out_lo) *reinterpret_cast<uint32_t*>(a.out_lo + at) = lo;
    }
}

// Row of the tables of mixed heads.
__device__ __forceinline__ int64_t table_row(const ChunkAttention& a, int sequence, int position) {
    return static_cast<int64_t>(sequence - a.first_sequence) * a.span + position - a.begin;
}
// Two adjacent weights (hi | lo << 16 each) as operand pairs.
__device__ __forceinline__ void unpack_weights(uint2 w, uint32_t& hi, uint32_t& lo) {
    hi = __byte_perm(w.x, w.y, 0x5410);
    lo = __byte_perm(w.x, w.y, 0x7632);
}
// What the attention kernels do: everything, or (mixed heads) the scores with their largest and sum, or the values under given weights.
enum ChunkPart { kWhole = 0, kScores = 1, kValues = 2 };

// 16-byte piece `chunk` of a tile row of COLUMNS values, swizzled by the row.
template <int COLUMNS> __device__ __forceinline__ uint32_t tile_offset(int row, int chunk) {
    return static_cast<uint32_t>(row * COLUMNS * 2 + ((chunk ^ (row & 7)) << 4));
}

// The rows and keys of one CTA of a longer pass: some positions of a sequence x some heads of a group; the keys that they see - `extra` kept
// positions or pooled blocks, then the positions from key_begin to key_end.
struct TileRows {
    const ChunkAttention& a;
    const ChunkParams& p;
    int sequence, head_tile, kv_head, first, count, slot, length, offset, last;
    int key_begin, key_end, extra, keys, in_slot, slot_start, ring_from, ring_at;
    __device__ __forceinline__ TileRows(const ChunkAttention& attention, int sequence_, int z, int offset_)
        : a(attention), p(attention.p), sequence(sequence_), head_tile(z % attention.head_tiles), kv_head(z / attention.head_tiles), offset(offset_) {
        first = __ldg(a.rows.first + sequence);
        count = __ldg(a.rows.first + sequence + 1) - first;
        slot = __ldg(a.rows.slot + sequence);
        length = a.rows.lengths[slot];
        last = min(offset + a.positions_per_tile, count);
        key_begin = p.first_seen(length + offset);
        key_end = length + last;
        extra = p.pool > 0 ? p.blocks_seen(key_end - 1) : min(p.keep, key_begin);
        keys = extra + key_end - key_begin;
        in_slot = p.appends_first(a.step) ? key_end : length;   // positions whose keys the slot holds
        slot_start = p.chunk_start(length);                     // position of the slot's entry 0
        ring_from = max(key_begin, p.keep);
        ring_at = p.window > 0 ? (ring_from - p.keep) % p.window : 0;
    }
    // row m of the tile: position inside the pass, and head
    __device__ __forceinline__ bool row(int m, int& position, int& head) const {
        position = offset + m / a.heads_per_tile;
        const int in_group = head_tile * a.heads_per_tile + m % a.heads_per_tile;
        head = kv_head * p.group + in_group;
        return m < a.positions_per_tile * a.heads_per_tile && position < last && in_group < p.group;
    }
    // entry of key n in the slot, or -1 - (row of the pass)
    __device__ __forceinline__ int place(int n) const {
        if (n < extra) return p.pool > 0 ? p.window + n : n;
        const int j = key_begin + n - extra;
        if (j >= in_slot) return -1 - (first + j - length);
        if (p.window == 0) return j - slot_start;
        if (j < p.keep) return j;
        const int at = ring_at + j - ring_from;   // (the slot holds less than a window from ring_from on)
        return p.keep + (at < p.window ? at : at - p.window);
    }
    // COLUMNS values of ROWS keys from key t0 on to shared memory, swizzled, by 128 threads
    template <int COLUMNS, int ROWS>
    __device__ __forceinline__ void fetch(uint32_t to, int t0, const void* cache, const void* workspace, int size) const {
        const auto* stored = static_cast<const __nv_bfloat16*>(cache) + (static_cast<int64_t>(slot) * p.kv_heads + kv_head) * p.entries * size;
        const auto* fresh = static_cast<const __nv_bfloat16*>(workspace) + kv_head * size;
#pragma unroll 4
        for (int c = threadIdx.x; c < ROWS * (COLUMNS / 8); c += 128) {
            const int n = c / (COLUMNS / 8), piece = c % (COLUMNS / 8);
            const bool live = t0 + n < keys && piece * 8 < size;
            const __nv_bfloat16* from = stored;
            if (live) {
                const int at = place(t0 + n);
                from = (at >= 0 ? stored + static_cast<int64_t>(at) * size : fresh + static_cast<int64_t>(-1 - at) * p.kv_heads * size) + piece * 8;
            }
            copy_async_16(to + tile_offset<COLUMNS>(n, piece), from, live);
        }
    }
    // ROWS x COLUMNS queries of the tile
    template <int COLUMNS, int ROWS> __device__ __forceinline__ void fetch_queries(uint32_t to) const {
        const auto* query = static_cast<const __nv_bfloat16*>(p.query);
        for (int c = threadIdx.x; c < ROWS * (COLUMNS / 8); c += 128) {
            const int m = c / (COLUMNS / 8), piece = c % (COLUMNS / 8);
            int position, head;
            const bool live = row(m, position, head) && piece * 8 < p.dim;
            copy_async_16(to + tile_offset<COLUMNS>(m, piece), live ? query + (static_cast<int64_t>(first + position) * p.heads + head) * p.dim + piece * 8 : query, live);
        }
    }
};
// the tiles with the most keys start first
__device__ __forceinline__ int tile_begin(const ChunkAttention& a) { return a.begin + (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * a.positions_per_tile; }

template <int DK, int DV, int PART = kWhole> struct ChunkShape {
    static constexpr int kWarps = 4, kThreads = kWarps * 32;
    static constexpr int kRows = 64;
    static constexpr int kKeys = PART != kWhole || DK + DV <= 256 ? 64 : 32;   // keys of a tile
    static constexpr int kKeyBytes = kKeys * DK * 2, kStageBytes = PART == kScores ? kKeyBytes : kKeyBytes + kKeys * DV * 2;
    static constexpr int kQueryBytes = kRows * DK * 2;
    static constexpr int kSmem = kQueryBytes + 2 * kStageBytes;
};

// PART kWhole or kScores
template <int DK, int DV, int PART>
__global__ void __launch_bounds__(128) chunk_mma_kernel(const __grid_constant__ ChunkAttention a) {
    using S = ChunkShape<DK, DV, PART>;
    extern __shared__ __align__(128) uint8_t smem[];
    const ChunkParams& p = a.p;
    uint8_t* ring = smem + S::kQueryBytes;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    grid_dependency_wait();
    grid_launch_dependents();
    const TileRows tile(a, a.first_sequence + blockIdx.y, blockIdx.z, tile_begin(a));
    if (tile.offset >= tile.count) return;
    const int tiles = (tile.keys + S::kKeys - 1) / S::kKeys;
    tile.fetch_queries<DK, S::kRows>(smem_u32(smem));
    auto fetch = [&](int t, int stage) {
        const uint32_t at = smem_u32(ring + stage * S::kStageBytes);
        tile.fetch<DK, S::kKeys>(at, t * S::kKeys, p.key_cache, p.key, p.dim);
        if constexpr (PART == kWhole) tile.fetch<DV, S::kKeys>(at + S::kKeyBytes, t * S::kKeys, p.value_cache, p.value, p.vdim);
    };
    fetch(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");

    const int row_base = warp * 16;
    // the two rows of this thread's fragments: which keys they see, [see_from, see_to) and the first see_extra
    int see_from[2], see_to[2], see_extra[2];
    float* table[2] = {nullptr, nullptr};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        int position, head;
        const bool live = tile.row(row_base + (lane >> 2) + i * 8, position, head);
        const int at = tile.length + position;
        see_from[i] = live ? tile.extra + p.first_seen(at) - tile.key_begin : 0;
        see_to[i] = live ? tile.extra + at + 1 - tile.key_begin : 0;
        see_extra[i] = !live ? 0 : p.pool > 0 ? p.blocks_seen(at) : p.keep;
        if (PART == kScores && live) table[i] = a.table + (table_row(a, tile.sequence, position) * p.heads + head) * a.pitch + (lane & 3) * 2;
    }
    // keys that every live row of this warp sees need no mask
    auto least = [&](const int (&v)[2]) { return -warp_max_int(-min(see_to[0] ? v[0] : INT32_MAX, see_to[1] ? v[1] : INT32_MAX)); };
    const int all_from = warp_max_int(max(see_to[0] ? see_from[0] : 0, see_to[1] ? see_from[1] : 0)), all_to = least(see_to), all_extra = least(see_extra);

    constexpr int NT = S::kKeys / 8, VT = PART == kWhole ? DV / 8 : 1;
    constexpr bool kHold = DK <= 128;      // query fragments stay in registers
    uint32_t q[kHold ? DK / 16 : 1][4];
    float o[VT][4];
#pragma unroll
    for (int v = 0; v < VT; ++v)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[v][i] = 0.0f;
    float top[2] = {-INFINITY, -INFINITY}, total[2] = {0.0f, 0.0f};
    const float scale2 = p.scale * kLog2e, cap2 = p.softcap * kLog2e, scale_by_cap = p.softcap > 0.0f ? p.scale / p.softcap : 0.0f;
    const uint32_t query_at = smem_u32(smem);
    const int query_row = row_base + (lane & 15);
    auto load_query = [&](uint32_t (&f)[4], int k) { ldsm_x4(f, query_at + tile_offset<DK>(query_row, k * 2 + (lane >> 4))); };

    for (int t = 0; t < tiles; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // the tile is here, and everyone is done with the stage that is filled next
        if (t + 1 < tiles) fetch(t + 1, (t + 1) & 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if constexpr (kHold) {
            if (t == 0) {
#pragma unroll
                for (int k = 0; k < DK / 16; ++k) load_query(q[k], k);
            }
        }
        const uint32_t key_tile = smem_u32(ring + (t & 1) * S::kStageBytes), value_tile = key_tile + S::kKeyBytes;
        float s[NT][4];
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) s[n][i] = 0.0f;
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
            if constexpr (!kHold) load_query(q[0], k);
            const uint32_t (&f)[4] = q[kHold ? k : 0];
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                uint32_t b[4];
                ldsm_x4(b, key_tile + tile_offset<DK>(n * 8 + (lane >> 4) * 8 + (lane & 7), k * 2 + ((lane >> 3) & 1)));
                mma_16816(s[n], f, b[0], b[1]);
                mma_16816(s[n + 1], f, b[2], b[3]);
            }
        }
        const int t0 = t * S::kKeys;
        const bool mask = t0 + S::kKeys > all_to || (t0 < all_from && t0 + S::kKeys > all_extra);
        float high[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                s[n][i] = p.softcap > 0.0f ? capped_score(s[n][i], scale_by_cap, cap2) : s[n][i] * scale2;
                if (mask) {
                    const int j = t0 + n * 8 + (lane & 3) * 2 + (i & 1);
                    if (j >= see_to[i >> 1] || (j < see_from[i >> 1] && j >= see_extra[i >> 1])) s[n][i] = -INFINITY;
                }
                high[i >> 1] = fmaxf(high[i >> 1], s[n][i]);
            }
        if constexpr (PART == kScores) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                if (!table[i]) continue;
#pragma unroll
                for (int n = 0; n < NT; ++n) *reinterpret_cast<float2*>(table[i] + t0 + n * 8) = make_float2(s[n][2 * i], s[n][2 * i + 1]);
            }
        }
        float base[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            high[i] = fmaxf(high[i], __shfl_xor_sync(0xffffffffu, high[i], 1));
            high[i] = fmaxf(high[i], __shfl_xor_sync(0xffffffffu, high[i], 2));
            const float next = fmaxf(top[i], high[i]);
            base[i] = next == -INFINITY ? 0.0f : next;
            const float factor = exp2_fast(top[i] - base[i]);
            top[i] = next;
            total[i] *= factor;
#pragma unroll
            for (int v = 0; v < VT; ++v) { o[v][2 * i] *= factor; o[v][2 * i + 1] *= factor; }
        }
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                s[n][i] = exp2_fast(s[n][i] - base[i >> 1]);
                total[i >> 1] += s[n][i];
            }
        if constexpr (PART == kScores) continue;
#pragma unroll
        for (int k = 0; k < NT / 2; ++k) {
            uint32_t hi[4], lo[4];
            pack_planes(s[2 * k][0], s[2 * k][1], hi[0], lo[0]);
            pack_planes(s[2 * k][2], s[2 * k][3], hi[1], lo[1]);
            pack_planes(s[2 * k + 1][0], s[2 * k + 1][1], hi[2], lo[2]);
            pack_planes(s[2 * k + 1][2], s[2 * k + 1][3], hi[3], lo[3]);
#pragma unroll
            for (int v = 0; v < VT; v += 2) {
                uint32_t b[4];
                ldsm_x4_trans(b, value_tile + tile_offset<DV>(k * 16 + (lane & 15), v + (lane >> 4)));
                mma_16816(o[v], hi, b[0], b[1]);
                mma_16816(o[v + 1], hi, b[2], b[3]);
                mma_16816(o[v], lo, b[0], b[1]);
                mma_16816(o[v + 1], lo, b[2], b[3]);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        total[i] += __shfl_xor_sync(0xffffffffu, total[i], 1);
        total[i] += __shfl_xor_sync(0xffffffffu, total[i], 2);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        int position, head;
        if (!tile.row(row_base + (lane >> 2) + i * 8, position, head)) continue;
        if constexpr (PART == kScores) {
            float* ml = a.table_ml + (table_row(a, tile.sequence, position) * p.heads + head) * 2;
            if ((lane & 3) == 0) { ml[0] = top[i]; ml[1] = total[i]; }
            continue;
        }
        const int row = tile.first + position;
        const float factor = head_gate(p, row, head) * denominator_factor(p, head, top[i], total[i]);
#pragma unroll
        for (int v = 0; v < VT; ++v) {
            const int column = v * 8 + (lane & 3) * 2;
            if (column < p.vdim) store_pair(a, row, head, column, o[v][2 * i] * factor, o[v][2 * i + 1] * factor);
        }
    }
}

// Longer passes of mixed heads: the values under the packed weights of the table.  The tiles are those of the scores.
template <int DV> struct ValueShape {
    static constexpr int kKeys = 64, kWeightBytes = 64 * (kKeys + 4) * 4, kStageBytes = kWeightBytes + kKeys * DV * 2, kSmem = 2 * kStageBytes;
};
template <int DV> __global__ void __launch_bounds__(128) talk_values_kernel(const __grid_constant__ ChunkAttention a) {
    using S = ValueShape<DV>;
    constexpr int kPitch = S::kKeys + 4;   // words between the rows of a weight tile
    extern __shared__ __align__(128) uint8_t smem[];
    const ChunkParams& p = a.p;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    grid_dependency_wait();
    grid_launch_dependents();
    const TileRows tile(a, a.first_sequence + blockIdx.y, blockIdx.z, tile_begin(a));
    if (tile.offset >= tile.count) return;
    const int tiles = (tile.keys + S::kKeys - 1) / S::kKeys;
    auto fetch = [&](int t, int stage) {
        const uint32_t at = smem_u32(smem + stage * S::kStageBytes);
#pragma unroll 4
        for (int c = threadIdx.x; c < 64 * (S::kKeys / 4); c += 128) {
            const int m = c / (S::kKeys / 4), piece = c % (S::kKeys / 4);
            int position, head;
            const bool live = tile.row(m, position, head);
            const float* from = live ? a.table + (table_row(a, tile.sequence, position) * p.heads + head) * a.pitch + t * S::kKeys + piece * 4 : a.table;
            copy_async_16(at + (m * kPitch + piece * 4) * 4, from, live);
        }
        tile.fetch<DV, S::kKeys>(at + S::kWeightBytes, t * S::kKeys, p.value_cache, p.value, p.vdim);
    };
    fetch(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    constexpr int VT = DV / 8;
    float o[VT][4];
#pragma unroll
    for (int v = 0; v < VT; ++v)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[v][i] = 0.0f;
    for (int t = 0; t < tiles; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // the tile is here, and everyone is done with the stage that is filled next
        if (t + 1 < tiles) fetch(t + 1, (t + 1) & 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const uint8_t* stage = smem + (t & 1) * S::kStageBytes;
        const uint32_t value_tile = smem_u32(stage + S::kWeightBytes);
        const uint32_t* weights = reinterpret_cast<const uint32_t*>(stage) + (warp * 16 + (lane >> 2)) * kPitch + (lane & 3) * 2;
#pragma unroll
        for (int k = 0; k < S::kKeys / 16; ++k) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int part = 0; part < 4; ++part)
                unpack_weights(*reinterpret_cast<const uint2*>(weights + (part & 1) * 8 * kPitch + k * 16 + (part >> 1) * 8), hi[part], lo[part]);
#pragma unroll
            for (int v = 0; v < VT; v += 2) {
                uint32_t b[4];
                ldsm_x4_trans(b, value_tile + tile_offset<DV>(k * 16 + (lane & 15), v + (lane >> 4)));
                mma_16816(o[v], hi, b[0], b[1]);
                mma_16816(o[v + 1], hi, b[2], b[3]);
                mma_16816(o[v], lo, b[0], b[1]);
                mma_16816(o[v + 1], lo, b[2], b[3]);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        int position, head;
        if (!tile.row(warp * 16 + (lane >> 2) + i * 8, position, head)) continue;
        const int row = tile.first + position;
        const float factor = head_gate(p, row, head);
#pragma unroll
        for (int v = 0; v < VT; ++v) {
            const int column = v * 8 + (lane & 3) * 2;
            if (column < p.vdim) store_pair(a, row, head, column, o[v][2 * i] * factor, o[v][2 * i + 1] * factor);
        }
    }
}

// Between the two: scores -> softmax weights, mixed over the heads -> packed bf16 planes, in place.  grid (blocks of keys, positions,
// sequences); a warp takes 32 keys of all heads at a time through the tensor cores: the matrix times the weights, both as two planes.
// Lane l loads the four keys from 4 (l / 4) on, one for each of four products of eight keys; so column c of product j is key 4 c + j,
// and every lane also ends with runs of four keys.  BLOCKS x 16 >= heads.
constexpr int kMixThreads = 128, kMixKeys = 512;
template <int BLOCKS> __global__ void __launch_bounds__(kMixThreads) talk_mix_kernel(const __grid_constant__ ChunkAttention a) {
    constexpr bool kHold = BLOCKS <= 2;   // the matrix stays in registers
    __shared__ uint32_t matrix[2][BLOCKS * BLOCKS * 4][32];   // planes of its fragments
    __shared__ float top[BLOCKS * 16], inverse[BLOCKS * 16];
    const ChunkParams& p = a.p;
    const int H = p.heads, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int c = threadIdx.x; c < BLOCKS * BLOCKS * 4 * 32; c += kMixThreads) {
        const int l = c & 31, part = (c >> 5) & 3, block = c >> 7;
        const int to = block / BLOCKS * 16 + (l >> 2) + (part & 1) * 8, from = block % BLOCKS * 16 + (l & 3) * 2 + (part >> 1) * 8;
        auto entry = [&](int g) { return to < H && g < H ? __ldg(p.talk + to * H + g) : 0.0f; };
        pack_planes(entry(from), entry(from + 1), matrix[0][block * 4 + part][l], matrix[1][block * 4 + part][l]);
    }
    grid_dependency_wait();
    grid_launch_dependents();
    const int sequence = a.first_sequence + blockIdx.z, position = a.begin + blockIdx.y;
    const int count = __ldg(a.rows.first + sequence + 1) - __ldg(a.rows.first + sequence);
    if (position >= count) return;
    int keys;
    if (a.step) keys = p.entries_seen(a.rows.lengths[__ldg(a.rows.slot + sequence)]);
    else keys = TileRows(a, sequence, 0, a.begin + (position - a.begin) / a.positions_per_tile * a.positions_per_tile).keys;
    keys = min((keys + 63) / 64 * 64, (static_cast<int>(blockIdx.x) + 1) * kMixKeys);   // (the tables are written in whole tiles)
    const int key0 = blockIdx.x * kMixKeys;
    if (key0 >= keys) return;
    const int64_t row = table_row(a, sequence, position) * H;
    for (int h = threadIdx.x; h < BLOCKS * 16; h += kMixThreads) {
        float high = -INFINITY, total = 0.0f;
        if (h < H) {
            const float* ml = a.table_ml + (row + h) * a.splits * 2;
            for (int s = 0; s < a.splits; ++s) high = fmaxf(high, ml[s * 2]);
            for (int s = 0; s < a.splits; ++s) total = fmaf(ml[s * 2 + 1], exp2_fast(ml[s * 2] - high), total);
        }
        top[h] = h < H ? high : 0.0f;
        inverse[h] = h < H ? 1.0f / total : 0.0f;
    }
    __syncthreads();
    uint32_t held[2][kHold ? BLOCKS * BLOCKS : 1][4];
    if constexpr (kHold) {
#pragma unroll
        for (int plane = 0; plane < 2; ++plane)
#pragma unroll
            for (int m = 0; m < BLOCKS * BLOCKS; ++m)
#pragma unroll
                for (int part = 0; part < 4; ++part) held[plane][m][part] = matrix[plane][m * 4 + part][lane];
    }
    const int head0 = (lane & 3) * 2;
    for (int n = key0 + warp * 32; n < keys; n += 4 * 32) {
        float* const at = a.table + row * a.pitch + n;
        uint32_t hi[BLOCKS][4][2], lo[BLOCKS][4][2];
        float4 score[BLOCKS][4];
#pragma unroll
        for (int k = 0; k < BLOCKS; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int h = k * 16 + head0 + (i & 1) + (i >> 1) * 8;
                score[k][i] = h < H ? __ldcg(reinterpret_cast<const float4*>(at + h * a.pitch + (lane >> 2) * 4)) : make_float4(-INFINITY, -INFINITY, -INFINITY, -INFINITY);
            }
#pragma unroll
        for (int k = 0; k < BLOCKS; ++k) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int h = k * 16 + head0 + (i & 1) + (i >> 1) * 8;
                const float high = top[h], factor = inverse[h];
                float4& w = score[k][i];
                w = make_float4(exp2_fast(w.x - high) * factor, exp2_fast(w.y - high) * factor, exp2_fast(w.z - high) * factor, exp2_fast(w.w - high) * factor);
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float4 u = score[k][2 * i], v = score[k][2 * i + 1];
                pack_planes(u.x, v.x, hi[k][0][i], lo[k][0][i]);
                pack_planes(u.y, v.y, hi[k][1][i], lo[k][1][i]);
                pack_planes(u.z, v.z, hi[k][2][i], lo[k][2][i]);
                pack_planes(u.w, v.w, hi[k][3][i], lo[k][3][i]);
            }
        }
#pragma unroll
        for (int m = 0; m < BLOCKS; ++m) {
            float c[4][4];
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) c[j][i] = 0.0f;
#pragma unroll
            for (int k = 0; k < BLOCKS; ++k) {
                uint32_t t_hi[4], t_lo[4];
#pragma unroll
                for (int part = 0; part < 4; ++part) {
                    t_hi[part] = kHold ? held[0][kHold ? m * BLOCKS + k : 0][part] : matrix[0][(m * BLOCKS + k) * 4 + part][lane];
                    t_lo[part] = kHold ? held[1][kHold ? m * BLOCKS + k : 0][part] : matrix[1][(m * BLOCKS + k) * 4 + part][lane];
                }
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    mma_16816(c[j], t_hi, hi[k][j][0], hi[k][j][1]);
                    mma_16816(c[j], t_hi, lo[k][j][0], lo[k][j][1]);
                    mma_16816(c[j], t_lo, hi[k][j][0], hi[k][j][1]);
                }
            }
            // (every lane's loads of these keys are behind the products)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int h = m * 16 + (lane >> 2) + half * 8;
                if (h >= H) continue;
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    uint32_t first_hi, first_lo, last_hi, last_lo;
                    pack_planes(c[0][half * 2 + i], c[1][half * 2 + i], first_hi, first_lo);
                    pack_planes(c[2][half * 2 + i], c[3][half * 2 + i], last_hi, last_lo);
                    *reinterpret_cast<uint4*>(at + h * a.pitch + (head0 + i) * 4) =
                        make_uint4(__byte_perm(first_hi, first_lo, 0x5410), __byte_perm(first_hi, first_lo, 0x7632), __byte_perm(last_hi, last_lo, 0x5410),
                                   __byte_perm(last_hi, last_lo, 0x7632));
                }
            }
        }
    }
}

// ---- steps ----------------------------------------------------------------------------------------------------------
constexpr int kStepKeys = 64, kStepBoxBytes = kStepKeys * 64 * 2;
constexpr int kStepConsumers = 128, kStepThreads = kStepConsumers + 32;
constexpr int kMaxStages = 6, kStepControlBytes = 256;
constexpr int kSmSmem = 227 * 1024;

struct StepItem { int sequence, slot, length, kv_head, head_tile, split; };

// Byte offset of 16-byte piece `piece` of a row inside boxes of 64 keys x 64 values, the piece swizzled by its row.
__device__ __forceinline__ uint32_t box_offset(int row, int piece) {
    return static_cast<uint32_t>((piece >> 3) * kStepBoxBytes + row * 128 + (((piece & 7) ^ (row & 7)) << 4));
}
__device__ __forceinline__ void step_consumers_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kStepConsumers) : "memory"); }

// CTAs that share an SM.
constexpr int step_residents(int columns) { return columns <= 128 ? 3 : columns <= 256 ? 2 : 1; }

// PART kScores leaves a tile's scores and their largest and sum in the tables, kValues takes packed weights from there.
template <int DK, int DV, int PART>
__global__ void __launch_bounds__(kStepThreads, step_residents(DK + DV)) chunk_step_kernel(const __grid_constant__ ChunkAttention a, const __grid_constant__ CUtensorMap key_map,
                                                                 const __grid_constant__ CUtensorMap value_map) {
    constexpr int kKeyBoxes = PART == kValues ? 0 : DK / 64, kValueBoxes = PART == kScores ? 0 : DV / 64, kStageBytes = (kKeyBoxes + kValueBoxes) * kStepBoxBytes;
    extern __shared__ __align__(128) uint8_t smem[];
    const ChunkParams& p = a.p;
    uint8_t* ring = smem + ((1024u - (smem_u32(smem) & 1023u)) & 1023u);   // swizzled boxes start on 1024-byte boundaries
    uint64_t* full = reinterpret_cast<uint64_t*>(ring + a.stages * kStageBytes);
    uint64_t* empty = full + kMaxStages;
    int* gave_up = reinterpret_cast<int*>(empty + kMaxStages);
    float* gates = reinterpret_cast<float*>(gave_up + 2);                                                     // [heads_per_tile]
    float* merge = reinterpret_cast<float*>(ring + a.stages * kStageBytes + kStepControlBytes);               // [warps][heads_per_tile][DV]
    float* merge_ml = merge + 4 * a.heads_per_tile * DV;                                                      // [warps][heads_per_tile][2]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < a.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], kStepConsumers / 32); }
        mbar_fence_init();
        *gave_up = 0;
        tma_prefetch_descriptor(&key_map);
        tma_prefetch_descriptor(&value_map);
    }
    __syncthreads();
    grid_dependency_wait();
    grid_launch_dependents();

    const int per_sequence = p.kv_heads * a.head_tiles * a.splits, items = a.rows.sequences * per_sequence;
    auto load_item = [&](int item) {
        StepItem it{};
        if (item < items) {
            it.sequence = item / per_sequence;
            const int rest = item - it.sequence * per_sequence, z = rest / a.splits;
            it.split = rest - z * a.splits;
            it.kv_head = z / a.head_tiles;
            it.head_tile = z - it.kv_head * a.head_tiles;
            it.slot = __ldg(a.rows.slot + it.sequence);
            it.length = a.rows.lengths[it.slot];
        }
        return it;
    };
    // tiles of an item: the slot holds the keys that the row sees, its own included, from entry 0 on
    auto keys_of = [&](const StepItem& it) { return p.entries_seen(it.length); };
    auto range_of = [&](const StepItem& it, int& tile0, int& tile1) {
        const int tiles = (keys_of(it) + kStepKeys - 1) / kStepKeys, per_split = (tiles + a.splits - 1) / a.splits;
        tile0 = it.split * per_split;
        tile1 = min(tiles, tile0 + per_split);
    };
    int stage = 0;
    uint32_t phase = 0;
    auto next_stage = [&] { if (++stage == a.stages) { stage = 0; phase ^= 1; } };
    StepItem now = load_item(blockIdx.x);

    if (warp == kStepConsumers / 32) {
        bool alive = true;
        for (int item = blockIdx.x; item < items && alive; item += gridDim.x) {
            const StepItem next = load_item(item + gridDim.x);
            int tile0, tile1;
            range_of(now, tile0, tile1);
            const int row0 = (now.slot * p.kv_heads + now.kv_head) * p.entries;
            for (int t = tile0; t < tile1; ++t) {
                if (!mbar_wait(&empty[stage], phase ^ 1)) {   // (passes at once in the first round)
                    if (lane == 0) atomicExch(a.status, B200_DEVICE_TIMEOUT);
                    alive = false;
                    break;
                }
                if (elect_one()) {
                    uint8_t* at = ring + stage * kStageBytes;
                    mbar_expect_tx(&full[stage], kStageBytes);
#pragma unroll
                    for (int b = 0; b < kKeyBoxes; ++b) tma_load_2d(at + b * kStepBoxBytes, &key_map, b * 64, row0 + t * kStepKeys, &full[stage]);
#pragma unroll
                    for (int b = 0; b < kValueBoxes; ++b)
                        tma_load_2d(at + (kKeyBoxes + b) * kStepBoxBytes, &value_map, b * 64, row0 + t * kStepKeys, &full[stage]);
                }
                __syncwarp();
                next_stage();
            }
            now = next;
        }
        return;
    }

    constexpr int VT = DV / 8;
    const float scale2 = p.scale * kLog2e, cap2 = p.softcap * kLog2e, scale_by_cap = p.softcap > 0.0f ? p.scale / p.softcap : 0.0f;
    const int own = warp * 16;   // this warp's keys of a tile
    for (int item = blockIdx.x; item < items; item += gridDim.x) {
        const int heads_here = min(a.heads_per_tile, p.group - now.head_tile * a.heads_per_tile);
        const int head0 = now.kv_head * p.group + now.head_tile * a.heads_per_tile;
        // queries as fragments: rows are the heads of the token
        uint32_t q[DK / 16][4];
        if constexpr (PART != kValues) {
            const auto* query = static_cast<const __nv_bfloat16*>(p.query) + (static_cast<int64_t>(now.sequence) * p.heads + head0) * p.dim;
#pragma unroll
            for (int k = 0; k < DK / 16; ++k)
#pragma unroll
                for (int part = 0; part < 4; ++part) {
                    const int m = (lane >> 2) + (part & 1) * 8, column = k * 16 + (lane & 3) * 2 + (part >> 1) * 8;
                    q[k][part] = m < heads_here && column < p.dim ? *reinterpret_cast<const uint32_t*>(query + m * p.dim + column) : 0u;
                }
        }
        const float gate = threadIdx.x < heads_here ? head_gate(p, now.sequence, head0 + threadIdx.x) : 0.0f;
        const StepItem next = load_item(item + gridDim.x);
        int tile0, tile1;
        range_of(now, tile0, tile1);
        const int keys = keys_of(now);
        float o[VT][4];
#pragma unroll
        for (int v = 0; v < VT; ++v)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[v][i] = 0.0f;
        float top[2] = {-INFINITY, -INFINITY}, total[2] = {0.0f, 0.0f};
        float* table[2] = {nullptr, nullptr};
        if constexpr (PART != kWhole) {
#pragma unroll
            for (int i = 0; i < 2; ++i)
                if ((lane >> 2) + i * 8 < heads_here)
                    table[i] = a.table + (static_cast<int64_t>(now.sequence) * p.heads + head0 + (lane >> 2) + i * 8) * a.pitch + own + (lane & 3) * 2;
        }
        for (int t = tile0; t < tile1; ++t) {
            if (!mbar_wait(&full[stage], phase)) {
                if (lane == 0) atomicExch(a.status, B200_DEVICE_TIMEOUT);
                *static_cast<volatile int*>(gave_up) = 1;
                break;
            }
            const uint32_t key_at = smem_u32(ring + stage * kStageBytes), value_at = key_at + kKeyBoxes * kStepBoxBytes;
            const int seen = keys - t * kStepKeys - own;   // keys of this warp's sixteen that exist
            if (PART == kScores && seen <= 0) {
#pragma unroll
                for (int i = 0; i < 2; ++i)
                    if (table[i]) {
                        *reinterpret_cast<float2*>(table[i] + t * kStepKeys) = make_float2(-INFINITY, -INFINITY);
                        *reinterpret_cast<float2*>(table[i] + t * kStepKeys + 8) = make_float2(-INFINITY, -INFINITY);
                    }
            }
            if (seen > 0) {
                uint32_t hi[4], lo[4];
                if constexpr (PART == kValues) {
#pragma unroll
                    for (int part = 0; part < 4; ++part)
                        unpack_weights(table[part & 1] ? __ldcg(reinterpret_cast<const uint2*>(table[part & 1] + t * kStepKeys + (part >> 1) * 8)) : make_uint2(0u, 0u),
                                       hi[part], lo[part]);
                } else {
                float s[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
#pragma unroll
                for (int k = 0; k < DK / 16; ++k) {
                    uint32_t b[4];
                    ldsm_x4(b, key_at + box_offset(own + (lane >> 4) * 8 + (lane & 7), k * 2 + ((lane >> 3) & 1)));
                    mma_16816(s[0], q[k], b[0], b[1]);
                    mma_16816(s[1], q[k], b[2], b[3]);
                }
                float high[2] = {-INFINITY, -INFINITY}, base[2];
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float score = p.softcap > 0.0f ? capped_score(s[n][i], scale_by_cap, cap2) : s[n][i] * scale2;
                        s[n][i] = n * 8 + (lane & 3) * 2 + (i & 1) < seen ? score : -INFINITY;
                        high[i >> 1] = fmaxf(high[i >> 1], s[n][i]);
                    }
                if constexpr (PART == kScores) {
#pragma unroll
                    for (int i = 0; i < 2; ++i)
                        if (table[i]) {
                            *reinterpret_cast<float2*>(table[i] + t * kStepKeys) = make_float2(s[0][2 * i], s[0][2 * i + 1]);
                            *reinterpret_cast<float2*>(table[i] + t * kStepKeys + 8) = make_float2(s[1][2 * i], s[1][2 * i + 1]);
                        }
                }
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    high[i] = fmaxf(high[i], __shfl_xor_sync(0xffffffffu, high[i], 1));
                    high[i] = fmaxf(high[i], __shfl_xor_sync(0xffffffffu, high[i], 2));
                    base[i] = fmaxf(top[i], high[i]);
                    const float factor = exp2_fast(top[i] - base[i]);
                    top[i] = base[i];
                    total[i] *= factor;
#pragma unroll
                    for (int v = 0; v < VT; ++v) { o[v][2 * i] *= factor; o[v][2 * i + 1] *= factor; }
                }
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        s[n][i] = exp2_fast(s[n][i] - base[i >> 1]);
                        total[i >> 1] += s[n][i];
                    }
                pack_planes(s[0][0], s[0][1], hi[0], lo[0]);
                pack_planes(s[0][2], s[0][3], hi[1], lo[1]);
                pack_planes(s[1][0], s[1][1], hi[2], lo[2]);
                pack_planes(s[1][2], s[1][3], hi[3], lo[3]);
                }
                // rows past the last key hold what the memory held: they must not reach the products, not even times zero
                uint32_t live[2] = {0xffffffffu, 0xffffffffu};
                if (seen < 16) {
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        const int left = seen - h * 8 - (lane & 3) * 2;
                        live[h] = left >= 2 ? 0xffffffffu : left == 1 ? 0x0000ffffu : 0u;
                    }
                }
#pragma unroll
                for (int v = 0; PART != kScores && v < VT; v += 2) {
                    uint32_t b[4];
                    ldsm_x4_trans(b, value_at + box_offset(own + (lane & 15), v + (lane >> 4)));
                    b[0] &= live[0]; b[1] &= live[1]; b[2] &= live[0]; b[3] &= live[1];
                    mma_16816(o[v], hi, b[0], b[1]);
                    mma_16816(o[v + 1], hi, b[2], b[3]);
                    mma_16816(o[v], lo, b[0], b[1]);
                    mma_16816(o[v + 1], lo, b[2], b[3]);
                }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[stage]);
            next_stage();
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            total[i] += __shfl_xor_sync(0xffffffffu, total[i], 1);
            total[i] += __shfl_xor_sync(0xffffffffu, total[i], 2);
        }
        // the warps' shares of the keys meet in shared memory
        step_consumers_sync();   // the item before has been read
        if (threadIdx.x < heads_here) gates[threadIdx.x] = gate;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int m = (lane >> 2) + i * 8;
            if (m >= heads_here) continue;
            const int at = warp * a.heads_per_tile + m;
#pragma unroll
            for (int v = 0; PART != kScores && v < VT; ++v)
                *reinterpret_cast<float2*>(merge + at * DV + v * 8 + (lane & 3) * 2) = make_float2(o[v][2 * i], o[v][2 * i + 1]);
            if ((lane & 3) == 0) { merge_ml[at * 2] = top[i]; merge_ml[at * 2 + 1] = total[i]; }
        }
        step_consumers_sync();
        if (*static_cast<volatile int*>(gave_up)) return;   // a tile never arrived: every consumer leaves here
        if constexpr (PART == kScores) {
            if (threadIdx.x < heads_here) {
                float best = -INFINITY, sum = 0.0f;
                for (int w = 0; w < 4; ++w) best = fmaxf(best, merge_ml[(w * a.heads_per_tile + threadIdx.x) * 2]);
                for (int w = 0; w < 4; ++w) {
                    const float* ml = merge_ml + (w * a.heads_per_tile + threadIdx.x) * 2;
                    sum = fmaf(ml[1], exp2_fast(ml[0] - (best == -INFINITY ? 0.0f : best)), sum);
                }
                float* to = a.table_ml + ((static_cast<int64_t>(now.sequence) * p.heads + head0 + threadIdx.x) * a.splits + now.split) * 2;
                to[0] = best;
                to[1] = sum;
            }
        }
        for (int c = threadIdx.x; PART != kScores && c < heads_here * (DV / 2); c += kStepConsumers) {
            const int m = c / (DV / 2), column = (c % (DV / 2)) * 2;
            if (column >= p.vdim) continue;
            float best = -INFINITY;
#pragma unroll
            for (int w = 0; w < 4; ++w) best = fmaxf(best, merge_ml[(w * a.heads_per_tile + m) * 2]);
            const float from = best == -INFINITY ? 0.0f : best;
            float x = 0.0f, y = 0.0f, sum = 0.0f;
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                const int at = w * a.heads_per_tile + m;
                const float factor = PART == kValues ? 1.0f : exp2_fast(merge_ml[at * 2] - from);
                const float2 v = *reinterpret_cast<const float2*>(merge + at * DV + column);
                x = fmaf(v.x, factor, x);
                y = fmaf(v.y, factor, y);
                sum = fmaf(merge_ml[at * 2 + 1], factor, sum);
            }
            const int head = head0 + m;
            if constexpr (PART == kValues) {   // the weights are finished: a share counts as it is
                best = 0.0f;
                sum = now.split == 0 ? 1.0f : 0.0f;
            }
            if (a.splits == 1) {
                const float factor = PART == kValues ? gates[m] : gates[m] * denominator_factor(p, head, from, sum);
                store_pair(a, now.sequence, head, column, x * factor, y * factor);
            } else {
                const int64_t part = (static_cast<int64_t>(now.sequence) * p.heads + head) * a.splits + now.split;
                *reinterpret_cast<float2*>(a.partial + part * p.vdim + column) = make_float2(x, y);
                if (column == 0) { a.partial_ml[part * 2] = best; a.partial_ml[part * 2 + 1] = sum; }
            }
        }
        now = next;
    }
}

// One CTA per (head, row): the splits' (max, sum, unscaled accumulator), and the gate.
__global__ void __launch_bounds__(64) chunk_combine_kernel(const __grid_constant__ ChunkAttention a) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int head = blockIdx.x, row = blockIdx.y;
    const int64_t at = (static_cast<int64_t>(row) * a.p.heads + head) * a.splits;
    float best = -INFINITY, total = 0.0f;
    for (int s = 0; s < a.splits; ++s) best = fmaxf(best, a.partial_ml[(at + s) * 2]);
    for (int s = 0; s < a.splits; ++s) total = fmaf(a.partial_ml[(at + s) * 2 + 1], exp2_fast(a.partial_ml[(at + s) * 2] - best), total);
    const float factor = head_gate(a.p, row, head) * denominator_factor(a.p, head, best, total);
    for (int c = threadIdx.x; c < a.p.vdim; c += blockDim.x) {
        float v = 0.0f;
        for (int s = 0; s < a.splits; ++s) v = fmaf(a.partial[(at + s) * a.p.vdim + c], exp2_fast(a.partial_ml[(at + s) * 2] - best), v);
        if (a.p.gate_values) v *= value_gate(a.p, row, head, c);
        store_forms(v * factor, row * a.out_stride + head * a.p.vdim + c, a.out, a.out_hi, a.out_lo);
    }
}

constexpr int kGenericThreads = 128, kGenericKeys = 128;

// The keys and values of one row as the plain kernels walk them: kept positions or pooled blocks, then the run up to the row itself.
template <class T> struct RowKeys {
    const ChunkParams& p;
    int slot, first, length, extra, begin, count, stored_end;
    __device__ __forceinline__ RowKeys(const ChunkAttention& a, const RowPlace& place)
        : p(a.p), slot(place.slot), first(__ldg(a.rows.first + place.sequence)), length(a.rows.lengths[place.slot]), extra(a.p.before_run(place.position)),
          begin(a.p.first_seen(place.position)), count(extra + place.position + 1 - begin), stored_end(a.p.appends_first(a.step) ? place.position + 1 : length) {}
    __device__ __forceinline__ const T* at(const void* cache, const void* rows, int size, int kv_head, int n) const {
        if (n < extra) return static_cast<const T*>(cache) + p.entry_at(slot, kv_head, p.pool > 0 ? p.window + n : n) * size;
        const int j = begin + n - extra;
        return j < stored_end ? static_cast<const T*>(cache) + p.entry(slot, kv_head, j) * size
                              : static_cast<const T*>(rows) + (static_cast<int64_t>(first + j - length) * p.kv_heads + kv_head) * size;
    }
    __device__ __forceinline__ const T* key(int kv_head, int n) const { return at(p.key_cache, p.key, p.dim, kv_head, n); }
    __device__ __forceinline__ const T* value(int kv_head, int n) const { return at(p.value_cache, p.value, p.vdim, kv_head, n); }
};

// grid (heads, rows): f32 FMAs over keys of either dtype
template <class T> __global__ void __launch_bounds__(kGenericThreads) chunk_generic_kernel(const __grid_constant__ ChunkAttention a) {
    extern __shared__ __align__(16) float sm[];   // query [dim], accumulator [vdim], weights [keys], scratch [32]
    const ChunkParams& p = a.p;
    float* query = sm;
    float* acc = query + p.dim;
    float* w = acc + p.vdim;
    float* scratch = w + kGenericKeys;
    grid_dependency_wait();
    grid_launch_dependents();
    const int head = blockIdx.x, row = blockIdx.y, kv_head = head / p.group, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const RowKeys<T> keys(a, row_place(a.rows, row));
    for (int c = threadIdx.x; c < p.dim; c += kGenericThreads)
        query[c] = load_as_f32(static_cast<const T*>(p.query), (static_cast<int64_t>(row) * p.heads + head) * p.dim + c);
    for (int c = threadIdx.x; c < p.vdim; c += kGenericThreads) acc[c] = 0.0f;
    float top = -INFINITY, total = 0.0f;
    for (int k0 = 0; k0 < keys.count; k0 += kGenericKeys) {
        const int n = min(kGenericKeys, keys.count - k0);
        __syncthreads();
        for (int j = warp; j < n; j += kGenericThreads / 32) {
            const T* key = keys.key(kv_head, k0 + j);
            float dot = 0.0f;
            for (int c = lane; c < p.dim; c += 32) dot = fmaf(query[c], load_as_f32(key, c), dot);
            dot = warp_sum(dot);
            if (lane == 0) w[j] = p.softcap > 0.0f ? p.softcap * tanhf(dot * p.scale / p.softcap) : dot * p.scale;
        }
        __syncthreads();
        float high = -INFINITY;
        for (int j = 0; j < n; ++j) high = fmaxf(high, w[j]);
        const float next = fmaxf(top, high), factor = expf(top - next);
        __syncthreads();
        if (threadIdx.x < n) w[threadIdx.x] = expf(w[threadIdx.x] - next);
        const float sum = block_sum(threadIdx.x < n ? w[threadIdx.x] : 0.0f, scratch);
        total = total * factor + sum;
        top = next;
        for (int c = threadIdx.x; c < p.vdim; c += kGenericThreads) {
            float v = acc[c] * factor;
            for (int j = 0; j < n; ++j) v = fmaf(w[j], load_as_f32(keys.value(kv_head, k0 + j), c), v);
            acc[c] = v;
        }
    }
    if (p.sink) {
        const float sink = __ldg(p.sink + head), high = fmaxf(top, sink), factor = expf(top - high);
        for (int c = threadIdx.x; c < p.vdim; c += kGenericThreads) acc[c] *= factor;
        total = fmaf(total, factor, expf(sink - high));
    }
    const float scale = head_gate(p, row, head) / total;
    for (int c = threadIdx.x; c < p.vdim; c += kGenericThreads)
        store_forms(acc[c] * (p.gate_values ? scale * value_gate(p, row, head, c) : scale), row * a.out_stride + head * p.vdim + c, a.out, a.out_hi, a.out_lo);
}

// Mixed heads, f32 FMAs: one CTA per row, all heads together.  A first sweep over the keys finds every head's largest score and sum, a
// second one the weights, mixed, and the values under them.
constexpr int kTalkThreads = 256, kTalkKeys = 64;
size_t talk_generic_bytes(const ChunkParams& p) {
    return (static_cast<size_t>(p.heads) * (p.dim + p.vdim + 2 * kTalkKeys + p.heads + 2)) * sizeof(float);
}
template <class T> __global__ void __launch_bounds__(kTalkThreads) talk_generic_kernel(const __grid_constant__ ChunkAttention a) {
    extern __shared__ __align__(16) float sm[];
    const ChunkParams& p = a.p;
    const int H = p.heads;
    float* query = sm;                        // [H][dim]
    float* acc = query + H * p.dim;           // [H][vdim]
    float* score = acc + H * p.vdim;          // [H][keys]
    float* mixed = score + H * kTalkKeys;     // [H][keys]
    float* talk = mixed + H * kTalkKeys;      // [H][H]
    float* top = talk + H * H;                // [H]
    float* total = top + H;                   // [H]
    grid_dependency_wait();
    grid_launch_dependents();
    const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const RowKeys<T> keys(a, row_place(a.rows, row));
    for (int c = threadIdx.x; c < H * p.dim; c += kTalkThreads) query[c] = load_as_f32(static_cast<const T*>(p.query), static_cast<int64_t>(row) * H * p.dim + c);
    for (int c = threadIdx.x; c < H * p.vdim; c += kTalkThreads) acc[c] = 0.0f;
    for (int c = threadIdx.x; c < H * H; c += kTalkThreads) talk[c] = p.talk[c];
    for (int h = threadIdx.x; h < H; h += kTalkThreads) { top[h] = -INFINITY; total[h] = 0.0f; }
    auto scores = [&](int k0, int n) {   // a warp per key and kv head, its heads one after the other
        for (int u = warp; u < n * p.kv_heads; u += kTalkThreads / 32) {
            const int j = u / p.kv_heads, kv_head = u - j * p.kv_heads;
            const T* key = keys.key(kv_head, k0 + j);
            for (int h = kv_head * p.group; h < (kv_head + 1) * p.group; ++h) {
                float dot = 0.0f;
                for (int c = lane; c < p.dim; c += 32) dot = fmaf(query[h * p.dim + c], load_as_f32(key, c), dot);
                dot = warp_sum(dot);
                if (lane == 0) score[h * kTalkKeys + j] = p.softcap > 0.0f ? p.softcap * tanhf(dot * p.scale / p.softcap) : dot * p.scale;
            }
        }
    };
    for (int k0 = 0; k0 < keys.count; k0 += kTalkKeys) {
        const int n = min(kTalkKeys, keys.count - k0);
        __syncthreads();
        scores(k0, n);
        __syncthreads();
        for (int h = warp; h < H; h += kTalkThreads / 32) {
            float high = top[h];
            for (int j = lane; j < n; j += 32) high = fmaxf(high, score[h * kTalkKeys + j]);
            high = warp_max(high);
            float sum = 0.0f;
            for (int j = lane; j < n; j += 32) sum += expf(score[h * kTalkKeys + j] - high);
            sum = warp_sum(sum);
            if (lane == 0) {
                total[h] = total[h] * expf(top[h] - high) + sum;
                top[h] = high;
            }
        }
    }
    for (int k0 = 0; k0 < keys.count; k0 += kTalkKeys) {
        const int n = min(kTalkKeys, keys.count - k0);
        __syncthreads();
        scores(k0, n);
        __syncthreads();
        for (int u = threadIdx.x; u < H * n; u += kTalkThreads) {
            const int h = u / n, at = h * kTalkKeys + u - h * n;
            score[at] = expf(score[at] - top[h]) / total[h];
        }
        __syncthreads();
        for (int u = threadIdx.x; u < H * n; u += kTalkThreads) {
            const int h = u / n, j = u - h * n;
            float sum = 0.0f;
            for (int g = 0; g < H; ++g) sum = fmaf(talk[h * H + g], score[g * kTalkKeys + j], sum);
            mixed[h * kTalkKeys + j] = sum;
        }
        __syncthreads();
        for (int c = threadIdx.x; c < H * p.vdim; c += kTalkThreads) {
            const int h = c / p.vdim, d = c - h * p.vdim;
            float v = acc[c];
            for (int j = 0; j < n; ++j) v = fmaf(mixed[h * kTalkKeys + j], load_as_f32(keys.value(h / p.group, k0 + j), d), v);
            acc[c] = v;
        }
    }
    __syncthreads();
    for (int c = threadIdx.x; c < H * p.vdim; c += kTalkThreads) {
        const int h = c / p.vdim, d = c - h * p.vdim;
        const float factor = p.gate_values ? p.out_scale * value_gate(p, row, h, d) : head_gate(p, row, h);
        store_forms(acc[c] * factor, row * a.out_stride + c, a.out, a.out_hi, a.out_lo);
    }
}

bool chunk_takes_mma(const ChunkParams& p, int dtype, int64_t out_stride) {
    return dtype == B200_BF16 && p.dim % 8 == 0 && p.vdim % 8 == 0 && p.dim <= 256 && p.vdim <= 256 && (out_stride & 1) == 0
        && (!p.gate_values || ((p.stride & 1) == 0 && (reinterpret_cast<uintptr_t>(p.projected) & 7) == 0))
        && ((reinterpret_cast<uintptr_t>(p.key_cache) | reinterpret_cast<uintptr_t>(p.value_cache)) & 15) == 0;
}

// Splits of a step's keys over CTAs: enough for two CTAs per SM, at least two tiles each.
int chunk_splits(const ChunkParams& p, int sequences, int max_length, int sms) {
    const int heads_per_tile = std::min(p.group, 16), items = sequences * p.kv_heads * ((p.group + heads_per_tile - 1) / heads_per_tile);
    const int keys = std::min(p.entries, max_length), tiles = (keys + 63) / 64;
    return std::max(1, std::min({(2 * sms + items - 1) / items, tiles / 2, 32}));
}

// grid of the tiles of the positions [begin, begin + span) of `sequences` sequences
dim3 tile_grid(const ChunkAttention& a, int sequences) {
    return dim3(static_cast<unsigned>((a.span + a.positions_per_tile - 1) / a.positions_per_tile), static_cast<unsigned>(sequences),
                static_cast<unsigned>(a.p.kv_heads * a.head_tiles));
}
template <int DK, int DV, int PART = kWhole> int launch_chunk_mma(const ChunkAttention& a, int sequences, cudaStream_t stream) {
    constexpr int kSmem = ChunkShape<DK, DV, PART>::kSmem;
    auto kernel = chunk_mma_kernel<DK, DV, PART>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem));
    return cuda_status(launch_dependent(kernel, tile_grid(a, sequences), dim3(128), kSmem, stream, a), "chunk_mma_kernel launch");
}
template <int DV> int launch_talk_values(const ChunkAttention& a, int sequences, cudaStream_t stream) {
    auto kernel = talk_values_kernel<DV>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, ValueShape<DV>::kSmem));
    return cuda_status(launch_dependent(kernel, tile_grid(a, sequences), dim3(128), ValueShape<DV>::kSmem, stream, a), "talk_values_kernel launch");
}
int launch_talk_mix(const ChunkAttention& a, int sequences, cudaStream_t stream) {
    auto kernel = a.p.heads <= 16 ? talk_mix_kernel<1> : a.p.heads <= 32 ? talk_mix_kernel<2> : a.p.heads <= 48 ? talk_mix_kernel<3> : talk_mix_kernel<4>;
    const dim3 grid(static_cast<unsigned>((a.pitch + kMixKeys - 1) / kMixKeys), static_cast<unsigned>(a.span), static_cast<unsigned>(sequences));
    return cuda_status(launch_dependent(kernel, grid, dim3(kMixThreads), 0, stream, a), "talk_mix_kernel launch");
}

int encode_slots(CUtensorMap* map, const void* base, int64_t rows, int columns) {
    encode_tiled_fn encode = tensor_map_encoder();
    if (!encode) { set_error("cuTensorMapEncodeTiled is not available from this driver"); return B200_NO_DEVICE; }
    const cuuint64_t dims[2] = {static_cast<cuuint64_t>(columns), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[1] = {static_cast<cuuint64_t>(columns) * 2};
    const cuuint32_t box[2] = {64, kStepKeys};
    const cuuint32_t element_strides[2] = {1, 1};
    const CUresult result = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, element_strides,
                                   CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (result != CUDA_SUCCESS) { set_error("cuTensorMapEncodeTiled(slots) failed with %d", static_cast<int>(result)); return B200_BAD_ARGUMENT; }
    return B200_OK;
}

template <int DK, int DV, int PART = kWhole> int launch_chunk_step(ChunkAttention a, int sms, cudaStream_t stream) {
    const ChunkParams& p = a.p;
    alignas(64) CUtensorMap keys, values;
    const int64_t rows = static_cast<int64_t>(p.slots) * p.kv_heads * p.entries;
    if (rows > INT32_MAX) { set_error("grouped attention: the slots hold more than 2^31 rows"); return B200_UNSUPPORTED; }
    int status = encode_slots(&keys, p.key_cache, rows, p.dim);
    if (status == B200_OK) status = encode_slots(&values, p.value_cache, rows, p.vdim);
    if (status != B200_OK) return status;
    const int stage_bytes = ((PART == kValues ? 0 : DK) + (PART == kScores ? 0 : DV)) / 64 * kStepBoxBytes, merge_bytes = 4 * a.heads_per_tile * (DV + 2) * 4, fixed = 1024 + kStepControlBytes + merge_bytes;
    int resident = step_residents(DK + DV) + 1;
    do a.stages = std::min((kSmSmem / --resident - 1024 - fixed) / stage_bytes, kMaxStages);
    while (a.stages < 2 && resident > 1);
    const int smem = fixed + a.stages * stage_bytes;
    auto kernel = chunk_step_kernel<DK, DV, PART>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    const int64_t items = static_cast<int64_t>(a.rows.sequences) * p.kv_heads * a.head_tiles * a.splits;
    if (items > INT32_MAX) { set_error("grouped attention: too many sequences and heads in one pass"); return B200_UNSUPPORTED; }
    return cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(std::min<int64_t>(items, resident * sms))), dim3(kStepThreads), smem, stream, a, keys,
                                        values), "chunk_step_kernel launch");
}

// The smallest pair of compiled head sizes that holds both.
template <class Launch> int pick_chunk_sizes(const ChunkParams& p, Launch&& launch) {
    using std::integral_constant;
    if (p.dim <= 64 && p.vdim <= 64) return launch(integral_constant<int, 64>{}, integral_constant<int, 64>{});
    if (p.dim <= 64 && p.vdim <= 128) return launch(integral_constant<int, 64>{}, integral_constant<int, 128>{});
    if (p.dim <= 128 && p.vdim <= 64) return launch(integral_constant<int, 128>{}, integral_constant<int, 64>{});
    if (p.dim <= 128 && p.vdim <= 128) return launch(integral_constant<int, 128>{}, integral_constant<int, 128>{});
    if (p.dim <= 192 && p.vdim <= 128) return launch(integral_constant<int, 192>{}, integral_constant<int, 128>{});
    return launch(integral_constant<int, 256>{}, integral_constant<int, 256>{});
}

// The smallest compiled size that holds one.
template <class Launch> int pick_head_size(int size, Launch&& launch) {
    using std::integral_constant;
    if (size <= 64) return launch(integral_constant<int, 64>{});
    if (size <= 128) return launch(integral_constant<int, 128>{});
    return launch(integral_constant<int, 256>{});
}

// Mixed heads: positions and sequences whose tables are filled at a time; longer passes go in portions.  (Portions whose tables stay in L2
// leave the SMs half empty and are slower than tables that do not.)
constexpr size_t kTableBytes = size_t{768} << 20;
constexpr int kMostMixedHeads = 64;   // (talk_mix_kernel)
struct TalkPlan { int64_t pitch; int span, sequences; };
TalkPlan talk_plan(const ChunkParams& p, int sequences, int max_count, int max_length) {
    const bool step = max_count == 1;
    const int tile = step ? 1 : 64 / std::min(p.group, 64);
    int64_t keys = max_length;
    if (p.window > 0) keys = std::min<int64_t>(keys, static_cast<int64_t>(p.window) + tile - 1) + (p.pool > 0 ? max_length / p.pool : p.keep);
    TalkPlan plan;
    plan.pitch = (keys + 63) / 64 * 64;
    plan.span = step ? 1 : (max_count + tile - 1) / tile * tile;
    plan.sequences = sequences;
    if (step) return plan;
    const size_t per_tile = static_cast<size_t>(tile) * p.heads * static_cast<size_t>(plan.pitch) * 4;
    const size_t tiles = std::max<size_t>(1, (p.table_bytes ? p.table_bytes : kTableBytes) / per_tile);
    plan.sequences = static_cast<int>(std::min<size_t>(static_cast<size_t>(sequences), tiles));
    plan.span = static_cast<int>(std::min<size_t>(static_cast<size_t>(plan.span), tiles / static_cast<size_t>(plan.sequences) * static_cast<size_t>(tile)));
    return plan;
}
size_t talk_table_words(const ChunkParams& p, const TalkPlan& plan) { return static_cast<size_t>(plan.sequences) * plan.span * p.heads * static_cast<size_t>(plan.pitch); }
size_t talk_scratch_bytes(const ChunkParams& p, const TalkPlan& plan, int splits) {
    const size_t rows = static_cast<size_t>(plan.sequences) * plan.span * p.heads;
    return (talk_table_words(p, plan) + rows * splits * 2 + (splits > 1 ? rows * splits * (p.vdim + 2) : 0)) * sizeof(float);
}
bool talk_takes_mma(const ChunkParams& p, int dtype, int64_t out_stride) {
    return p.talk && p.heads <= kMostMixedHeads && chunk_takes_mma(p, dtype, out_stride);
}

// scores -> mixed softmax weights -> values
int launch_talk(ChunkAttention a, int max_length, void* scratch, size_t scratch_bytes, int sms, cudaStream_t stream) {
    const ChunkParams& p = a.p;
    const TalkPlan plan = talk_plan(p, a.rows.sequences, a.rows.max_count, max_length);
    const size_t need = talk_scratch_bytes(p, plan, a.splits), rows = static_cast<size_t>(plan.sequences) * plan.span * p.heads;
    if (scratch_bytes < need || !scratch || (reinterpret_cast<uintptr_t>(scratch) & 15)) {
        set_error("b200_chunk_attention: scratch of %zu bytes, %zu needed", scratch_bytes, need);
        return B200_BAD_ARGUMENT;
    }
    a.pitch = plan.pitch;
    a.table = static_cast<float*>(scratch);
    a.table_ml = a.table + talk_table_words(p, plan);
    a.partial = a.table_ml + rows * a.splits * 2;
    a.partial_ml = a.partial + (a.splits > 1 ? rows * a.splits * p.vdim : 0);
    if (a.step) {
        a.span = 1;
        int status = pick_head_size(p.dim, [&](auto dk) { return launch_chunk_step<decltype(dk)::value, 64, kScores>(a, sms, stream); });
        if (status == B200_OK) status = launch_talk_mix(a, a.rows.sequences, stream);
        if (status == B200_OK) status = pick_head_size(p.vdim, [&](auto dv) { return launch_chunk_step<64, decltype(dv)::value, kValues>(a, sms, stream); });
        if (status == B200_OK && a.splits > 1)
            status = cuda_status(launch_dependent(chunk_combine_kernel, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(a.rows.rows)), dim3(64), 0, stream, a),
                                 "chunk_combine_kernel launch");
        return status;
    }
    for (int sequence = 0; sequence < a.rows.sequences; sequence += plan.sequences)
        for (int begin = 0; begin < a.rows.max_count; begin += plan.span) {
            const int sequences = std::min(plan.sequences, a.rows.sequences - sequence);
            a.first_sequence = sequence;
            a.begin = begin;
            a.span = plan.span;
            int status = pick_head_size(p.dim, [&](auto dk) { return launch_chunk_mma<decltype(dk)::value, 64, kScores>(a, sequences, stream); });
            if (status == B200_OK) status = launch_talk_mix(a, sequences, stream);
            if (status == B200_OK) status = pick_head_size(p.vdim, [&](auto dv) { return launch_talk_values<decltype(dv)::value>(a, sequences, stream); });
            if (status != B200_OK) return status;
        }
    return B200_OK;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_chunk_prepare(const b200_chunk_args* args, const b200_rows* pass, const b200_units* units, const b200_route* route, void* stream) {
    ChunkParams p;
    RowsView rows;
    if (!chunk_params(args, p) || !rows_view(pass, rows)) return B200_BAD_ARGUMENT;
    const bool step = rows.max_count == 1;
    if (!p.appends_first(step) && (!p.key || !p.value)) { set_error("b200_chunk_prepare: longer passes need key and value workspaces"); return B200_BAD_ARGUMENT; }
    Units u{};
    if (units && units->kind) {
        if (units->kind < 0 || units->kind > 2 || units->column < 0 || units->count < 0 || units->count > INT32_MAX || units->out_stride < units->count
            || units->column + units->count * (units->kind == 1 ? 2 : 1) > p.stride || (!units->out && !units->out_hi) || (units->out_hi && !units->out_lo)) {
            set_error("b200_chunk_prepare: inconsistent units");
            return B200_BAD_ARGUMENT;
        }
        u = Units{units->kind, units->column, static_cast<int>(units->count), units->out, static_cast<__nv_bfloat16*>(units->out_hi),
                  static_cast<__nv_bfloat16*>(units->out_lo), units->out_stride};
    }
    Route r{};
    if (route && route->experts) {
        if (!route_view(route, r) || route->column + route->experts > p.stride) {
            set_error("b200_chunk_prepare: inconsistent router");
            return B200_BAD_ARGUMENT;
        }
    }
    const int q = p.heads * p.dim, k = p.kv_heads * p.dim;
    auto aligned = [](const void* at) { return (reinterpret_cast<uintptr_t>(at) & 15) == 0; };
    auto aligned8 = [](const void* at) { return (reinterpret_cast<uintptr_t>(at) & 7) == 0; };
    const bool vector = p.dim % 4 == 0 && p.vdim % 4 == 0 && (p.rotate_pairs || (p.rot_dims >> 1) % 4 == 0) && p.stride % 4 == 0 && aligned(p.projected) && aligned(p.q_norm)
        && aligned(p.k_norm) && aligned(p.q_bias) && aligned(p.k_bias) && aligned(p.query) && aligned(p.key) && aligned(p.value) && aligned(p.key_cache) && aligned(p.value_cache)
        && aligned(p.pool_state) && (p.rot_dims == 0 || (aligned(p.cosine) && aligned(p.sine))) && q % 4 == 0 && k % 4 == 0
        && (u.kind == 0 || (u.column % 4 == 0 && u.count % 4 == 0 && u.stride % 4 == 0 && aligned(u.out) && aligned8(u.out_hi) && aligned8(u.out_lo)));
    const dim3 grid(static_cast<unsigned>(rows.rows), static_cast<unsigned>(1 + (u.count + kUnitSlice - 1) / kUnitSlice));
    auto launch = [&](auto norm) {
        constexpr int kNorm = decltype(norm)::value;
        auto kernel = args->dtype == B200_BF16 ? (vector ? chunk_prepare_kernel<__nv_bfloat16, 4, kNorm> : chunk_prepare_kernel<__nv_bfloat16, 1, kNorm>)
                                               : (vector ? chunk_prepare_kernel<float, 4, kNorm> : chunk_prepare_kernel<float, 1, kNorm>);
        return cuda_status(launch_dependent(kernel, grid, dim3(kPrepareThreads), static_cast<size_t>(r.experts) * 4, as_stream(stream), p, rows, step, u, r),
                           "chunk_prepare_kernel launch");
    };
    switch (p.norm) {
    case B200_HEAD_NORM_NONE: return launch(std::integral_constant<int, B200_HEAD_NORM_NONE>{});
    case B200_HEAD_NORM_HEAD: return launch(std::integral_constant<int, B200_HEAD_NORM_HEAD>{});
    default: return launch(std::integral_constant<int, B200_HEAD_NORM_PROJECTION>{});
    }
}

extern "C" size_t b200_chunk_scratch_bytes(const b200_chunk_args* args, int64_t rows, int32_t sequences, int32_t max_count, int32_t max_length) {
    ChunkParams p;
    if (!chunk_params(args, p) || rows <= 0 || sequences <= 0 || (max_count != 1 && !p.talk)) return 0;
    int device = 0;
    if (cudaGetDevice(&device) != cudaSuccess) { cudaGetLastError(); device = -1; }
    const int splits = max_count == 1 ? chunk_splits(p, sequences, max_length, sm_count(device)) : 1;
    if (p.talk) return p.heads <= kMostMixedHeads ? talk_scratch_bytes(p, talk_plan(p, sequences, max_count, max_length), splits) : 0;
    return splits > 1 ? static_cast<size_t>(rows) * p.heads * splits * (p.vdim + 2) * sizeof(float) : 0;
}

extern "C" int b200_chunk_attention(const b200_chunk_args* args, const b200_rows* pass, int32_t max_length, void* scratch, size_t scratch_bytes,
                                    float* out, void* out_hi, void* out_lo, int64_t out_stride, void* stream) {
    ChunkAttention a{};
    if (!chunk_params(args, a.p) || !rows_view(pass, a.rows)) return B200_BAD_ARGUMENT;
    const ChunkParams& p = a.p;
    if ((!out && !out_hi) || (out_hi && !out_lo) || out_stride < static_cast<int64_t>(p.heads) * p.vdim || max_length <= 0) {
        set_error("b200_chunk_attention: bad pointer or size");
        return B200_BAD_ARGUMENT;
    }
    cudaStream_t s = as_stream(stream);
    a.step = a.rows.max_count == 1;
    a.out = out; a.out_hi = static_cast<__nv_bfloat16*>(out_hi); a.out_lo = static_cast<__nv_bfloat16*>(out_lo); a.out_stride = out_stride;
    a.splits = 1;
    if (!p.appends_first(a.step) && (!p.key || !p.value)) { set_error("b200_chunk_attention: longer passes need key and value workspaces"); return B200_BAD_ARGUMENT; }
    int status = B200_OK;
    if (!a.step && p.pool > 0) {
        const bool quads = p.dim % 4 == 0 && p.vdim % 4 == 0
            && ((reinterpret_cast<uintptr_t>(p.key) | reinterpret_cast<uintptr_t>(p.value) | reinterpret_cast<uintptr_t>(p.key_cache)
                 | reinterpret_cast<uintptr_t>(p.value_cache) | reinterpret_cast<uintptr_t>(p.pool_state)) & 15) == 0;
        auto pool = args->dtype == B200_BF16 ? (quads ? chunk_pool_kernel<__nv_bfloat16, 4> : chunk_pool_kernel<__nv_bfloat16, 1>)
                                             : (quads ? chunk_pool_kernel<float, 4> : chunk_pool_kernel<float, 1>);
        if (a.rows.sequences > 65535) { set_error("grouped attention: at most 65535 sequences in one pass"); return B200_UNSUPPORTED; }
        const int columns = p.kv_heads * (p.dim + p.vdim), per_block = kPoolThreads * (quads ? 4 : 1);
        const dim3 grid(static_cast<unsigned>(a.rows.max_count / p.pool + 2), static_cast<unsigned>(a.rows.sequences), static_cast<unsigned>((columns + per_block - 1) / per_block));
        status = cuda_status(launch_dependent(pool, grid, dim3(kPoolThreads), 0, s, p, a.rows), "chunk_pool_kernel launch");
        if (status != B200_OK) return status;
    }
    if (p.talk && !talk_takes_mma(p, args->dtype, out_stride)) {
        const size_t smem = talk_generic_bytes(p);
        auto kernel = args->dtype == B200_BF16 ? talk_generic_kernel<__nv_bfloat16> : talk_generic_kernel<float>;
        if (smem > 220 * 1024) { set_error("mixed heads: %d heads of %d and %d are too large", p.heads, p.dim, p.vdim); return B200_UNSUPPORTED; }
        B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        status = cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(a.rows.rows)), dim3(kTalkThreads), smem, s, a), "talk_generic_kernel launch");
    } else if (chunk_takes_mma(p, args->dtype, out_stride)) {
        int device = 0;
        B200_CUDA(cudaGetDevice(&device));
        const int most = a.step ? 16 : 64;
        a.heads_per_tile = std::min(p.group, most);
        a.head_tiles = (p.group + a.heads_per_tile - 1) / a.heads_per_tile;
        a.positions_per_tile = a.step ? 1 : most / a.heads_per_tile;
        if (a.step) {
            a.splits = chunk_splits(p, a.rows.sequences, max_length, sm_count(device));
            const size_t need = a.splits > 1 && !p.talk ? static_cast<size_t>(a.rows.rows) * p.heads * a.splits * (p.vdim + 2) * sizeof(float) : 0;
            if (scratch_bytes < need || (need && !scratch)) { set_error("b200_chunk_attention: scratch of %zu bytes, %zu needed", scratch_bytes, need); return B200_BAD_ARGUMENT; }
            a.partial = static_cast<float*>(scratch);
            a.partial_ml = a.partial + static_cast<int64_t>(a.rows.rows) * p.heads * a.splits * p.vdim;
        }
        if (a.rows.sequences > 65535 || p.kv_heads * a.head_tiles > 65535) {
            set_error("grouped attention: at most 65535 sequences and head tiles in one pass");
            return B200_UNSUPPORTED;
        }
        a.status = device_status_word(device);
        if (!a.status) { set_error("the device status word could not be allocated"); return B200_NO_DEVICE; }
        const int sms = sm_count(device);
        a.span = a.rows.max_count;
        status = p.talk ? launch_talk(a, max_length, scratch, scratch_bytes, sms, s) : pick_chunk_sizes(p, [&](auto dk, auto dv) {
            constexpr int kDim = decltype(dk)::value, kValueDim = decltype(dv)::value;
            return a.step ? launch_chunk_step<kDim, kValueDim>(a, sms, s) : launch_chunk_mma<kDim, kValueDim>(a, a.rows.sequences, s);
        });
        if (status == B200_OK && a.splits > 1 && !p.talk)
            status = cuda_status(launch_dependent(chunk_combine_kernel, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(a.rows.rows)), dim3(64), 0, s, a),
                                 "chunk_combine_kernel launch");
    } else {
        if (a.rows.rows > 65535) { set_error("grouped attention: at most 65535 rows in one pass"); return B200_UNSUPPORTED; }
        const size_t smem = (static_cast<size_t>(p.dim) + p.vdim + kGenericKeys + 32) * sizeof(float);
        auto kernel = args->dtype == B200_BF16 ? chunk_generic_kernel<__nv_bfloat16> : chunk_generic_kernel<float>;
        if (smem > 200 * 1024) { set_error("grouped attention: head sizes %d and %d are too large", p.dim, p.vdim); return B200_UNSUPPORTED; }
        B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        status = cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(a.rows.rows)), dim3(kGenericThreads), smem, s, a),
                             "chunk_generic_kernel launch");
    }
    if (status != B200_OK || p.appends_first(a.step)) return status;
    auto append = args->dtype == B200_BF16 ? chunk_append_kernel<__nv_bfloat16> : chunk_append_kernel<float>;
    return cuda_status(launch_dependent(append, dim3(static_cast<unsigned>(std::min(a.rows.rows, 1184))), dim3(128), 0, s, p, a.rows), "chunk_append_kernel launch");
}

extern "C" const char* b200_chunk_attention_kernel(const b200_chunk_args* args, int32_t max_count, int64_t out_stride) {
    ChunkParams p;
    if (!chunk_params(args, p)) return "";
    if (p.talk) return !talk_takes_mma(p, args->dtype, out_stride) ? "talk_generic_kernel" : max_count == 1 ? "chunk_step_kernel" : "talk_values_kernel";
    if (!chunk_takes_mma(p, args->dtype, out_stride)) return "chunk_generic_kernel";
    return max_count == 1 ? "chunk_step_kernel" : "chunk_mma_kernel";
}
