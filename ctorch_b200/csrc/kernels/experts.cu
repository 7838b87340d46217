// Mixture of experts: every slot (row, choice) adds expert(weight * row) or weight * expert(row), expert(x) = down gelu(up x) or
// down (silu(gate x) * (up x)) with gate and up rows interleaved.  A weight of the expert's input joins the row's norm factor in front of
// the activation; a weight of its result is applied where the choices of a row are added up.  Choices past the experts are identity
// experts: they add the weighted row itself and have no slots to sort.
//
//   * streamed: few slots, f32 weights, odd sizes.  expert_up_kernel and expert_down_kernel let every slot stream its expert's rows with
//     f32 FMAs; the down form adds the choices of a row and the residual itself.
//   * grouped: the slots are sorted by expert (expert_gather_kernel: planes of the rows copied into order, the list of row tiles
//     written), then expert_gemm_kernel multiplies tiles of up to 128 slots of ONE expert with its weights on the tensor cores
//     (persistent CTAs over the list, TMA operand ring, tcgen05, double-buffered accumulator, the row epilogues of the dense kernels);
//     only the 32-row boxes that hold slots are fetched, so a batch that gives every expert a few rows costs the weight stream.
//     expert_combine_kernel adds every row's results in the order of its choices: the sum does not depend on the sorting.  Where a norm
//     stands behind the mixture it finishes the row as well (sandwich.cuh).
#include "linear_rows.cuh"
#include "router.cuh"
#include "rows.cuh"
#include "sandwich.cuh"
#include "tcgen05.cuh"

#include <algorithm>

namespace b200 {
namespace {

struct ExpertParams {
    int experts, top, rows, in, ff;
    const void *up, *down;
    const int32_t* chosen;
    const float* weight;
    const float* x;
    const __nv_bfloat16 *x_hi, *x_lo;
    const float* sumsq_in;
    int parts_in;
    float eps;
    const float* residual;
    float* y;
    bool gated, weigh_results;
    int identity;
    SandwichView after;
    bool finishes;   // `after` is set
};

bool expert_params(const b200_experts* a, ExpertParams& p) {
    if (!a || a->experts <= 0 || a->experts > B200_MAX_EXPERTS || a->top <= 0 || a->rows <= 0 || a->in <= 0 || a->ff <= 0
        || a->rows * a->top > INT32_MAX || a->in > INT32_MAX || a->ff > INT32_MAX || a->experts * std::max(a->in, 2 * a->ff) > INT32_MAX || a->top > a->experts + a->identity || a->identity < 0
        || (a->weight_dtype != B200_F32 && a->weight_dtype != B200_BF16) || !a->up || !a->down || !a->chosen || !a->weight
        || (!a->x && (!a->x_hi || !a->x_lo)) || (a->parts_in > 0 && !a->sumsq_in) || a->parts_in < 0
        || (!a->y && !a->after)) {
        set_error("mixture of experts: bad pointer or size");
        return false;
    }
    p = ExpertParams{a->experts, a->top, static_cast<int>(a->rows), static_cast<int>(a->in), static_cast<int>(a->ff), a->up, a->down, a->chosen, a->weight,
                     a->x, static_cast<const __nv_bfloat16*>(a->x_hi), static_cast<const __nv_bfloat16*>(a->x_lo), a->sumsq_in, a->parts_in,
                     static_cast<float>(a->eps), a->residual, a->y, a->gated != 0, a->weigh_results != 0, a->identity, SandwichView{}, a->after != nullptr};
    if (a->after && !sandwich_view(a->after, p.after)) {
        set_error("mixture of experts: inconsistent norm behind the mixture");
        return false;
    }
    return true;
}

// Factor of a row: the split norm's scale (1 without one).
__device__ __forceinline__ float row_factor(const ExpertParams& p, int row) {
    float scale = 1.0f;
    if (p.parts_in > 0) {
        float total = 0.0f;
        for (int i = 0; i < p.parts_in; ++i) total += __ldg(p.sumsq_in + static_cast<int64_t>(i) * p.rows + row);
        scale = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(total, static_cast<float>(p.in)), p.eps)));
    }
    return scale;
}
// Factor of a slot's input: its row's, and the router's weight where that multiplies the input.
__device__ __forceinline__ float slot_scale(const ExpertParams& p, int slot) {
    return row_factor(p, slot / p.top) * (p.weigh_results ? 1.0f : __ldg(p.weight + slot));
}
__device__ __forceinline__ float row_value(const ExpertParams& p, int64_t at) {
    return p.x ? p.x[at] : __bfloat162float(p.x_hi[at]) + __bfloat162float(p.x_lo[at]);
}
// Weights of a row's identity choices together.
__device__ __forceinline__ float identity_weight(const ExpertParams& p, int row) {
    float total = 0.0f;
    if (p.identity > 0)
        for (int k = 0; k < p.top; ++k)
            if (__ldg(p.chosen + row * p.top + k) >= p.experts) total += __ldg(p.weight + row * p.top + k);
    return total;
}

// ---- streamed -------------------------------------------------------------------------------------------------------
constexpr int kStreamThreads = 256, kStreamWarps = kStreamThreads / 32;

// Dot products of F weight rows with a vector in shared memory, by one warp; every lane gets its share of the sums.
template <class W, bool VECTOR, int F>
__device__ __forceinline__ void dot_rows(const W* const (&w)[F], const float* x, int n, int lane, float (&acc)[F]) {
    if constexpr (VECTOR) {
        constexpr int kPer = 16 / sizeof(W);
#pragma unroll (F < 8 ? 8 / F : 1)
        for (int k = lane * kPer; k < n; k += 32 * kPer) {
            uint4 raw[F];
#pragma unroll
            for (int f = 0; f < F; ++f) raw[f] = load_stream_16(w[f] + k);
            float v[kPer];
#pragma unroll
            for (int i = 0; i < kPer; i += 4) {
                const float4 q = *reinterpret_cast<const float4*>(x + k + i);
                v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
            }
#pragma unroll
            for (int f = 0; f < F; ++f) {
                const uint32_t r[4] = {raw[f].x, raw[f].y, raw[f].z, raw[f].w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if constexpr (sizeof(W) == 2) acc[f] = fmaf(v[2 * i], bf16_lo(r[i]), fmaf(v[2 * i + 1], bf16_hi(r[i]), acc[f]));
                    else acc[f] = fmaf(v[i], __uint_as_float(r[i]), acc[f]);
                }
            }
        }
    } else {
        for (int k = lane; k < n; k += 32)
#pragma unroll
            for (int f = 0; f < F; ++f) acc[f] = fmaf(x[k], load_as_f32(w[f], k), acc[f]);
    }
}

// Asks for the CTA's weight rows [first, last) of an expert while the kernel before is still running.  The router's choice is older than
// that kernel in every plan; where it is not, a stale number (kept in range) only fetches rows in vain.  Worth it while the grid is about
// one CTA per SM (F = 1); later waves would only ask for what they are about to load.
template <class W> __device__ __forceinline__ void prefetch_rows(const W* matrix, int expert, int experts, int out, int in, int first, int last) {
    const int known = min(max(expert, 0), experts - 1);
    const auto* at = reinterpret_cast<const uint8_t*>(matrix + (static_cast<int64_t>(known) * out + first) * in);
    const int64_t bytes = static_cast<int64_t>(last - first) * in * static_cast<int>(sizeof(W));
    for (int64_t o = static_cast<int64_t>(threadIdx.x) * 128; o < bytes; o += kStreamThreads * 128) prefetch_l2(at + o);
}

// grid (slots, feature blocks): act[slot, f] = gelu(up_f . (scale * row)), or the gated unit of rows 2f and 2f + 1; F features per warp
template <class W, bool VECTOR, int F, bool GATED>
__global__ void __launch_bounds__(kStreamThreads) expert_up_kernel(const __grid_constant__ ExpertParams p, float* act) {
    constexpr int kPer = GATED ? 2 : 1, kRows = F * kPer;   // weight rows per feature, per warp
    extern __shared__ __align__(16) float x[];
    const int slot = blockIdx.x, row = slot / p.top, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int block0 = blockIdx.y * kStreamWarps * F, f0 = block0 + warp * F;
    if constexpr (F == 1) prefetch_rows(static_cast<const W*>(p.up), *static_cast<const volatile int32_t*>(p.chosen + slot), p.experts, p.ff * kPer, p.in, block0 * kPer, min(block0 + kStreamWarps * F, p.ff) * kPer);
    grid_dependency_wait();
    grid_launch_dependents();
    const int expert = *static_cast<const volatile int32_t*>(p.chosen + slot);
    if (expert >= p.experts) return;   // an identity expert
    const float scale = slot_scale(p, slot);
    const int64_t base = static_cast<int64_t>(row) * p.in;
    for (int c = threadIdx.x; c < p.in; c += kStreamThreads) x[c] = row_value(p, base + c) * scale;
    __syncthreads();
    if (f0 >= p.ff) return;
    const W* w[kRows];
    float acc[kRows];
#pragma unroll
    for (int f = 0; f < kRows; ++f) {
        w[f] = static_cast<const W*>(p.up) + (static_cast<int64_t>(expert) * p.ff * kPer + min(f0 * kPer + f, p.ff * kPer - 1)) * p.in;
        acc[f] = 0.0f;
    }
    dot_rows<W, VECTOR, kRows>(w, x, p.in, lane, acc);
#pragma unroll
    for (int f = 0; f < F; ++f) {
        float v;
        if constexpr (GATED) {
            const float gate = warp_sum(acc[2 * f]), up = warp_sum(acc[2 * f + 1]);
            v = silu_reference(gate) * up;
        } else {
            v = gelu_exact(warp_sum(acc[f]));
        }
        if (lane == f && f0 + f < p.ff) act[static_cast<int64_t>(slot) * p.ff + f0 + f] = v;
    }
}

// grid (rows, feature blocks): y = residual + sum over the choices of down . act
template <class W, bool VECTOR, int F> __global__ void __launch_bounds__(kStreamThreads) expert_down_kernel(const __grid_constant__ ExpertParams p, const float* act) {
    extern __shared__ __align__(16) float x[];
    const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int block0 = blockIdx.y * kStreamWarps * F, f0 = block0 + warp * F;
    for (int k = 0; F == 1 && k < p.top; ++k)
        prefetch_rows(static_cast<const W*>(p.down), *static_cast<const volatile int32_t*>(p.chosen + row * p.top + k), p.experts, p.in, p.ff, block0,
                      min(block0 + kStreamWarps * F, p.in));
    grid_dependency_wait();
    grid_launch_dependents();
    float sum[F];
#pragma unroll
    for (int f = 0; f < F; ++f) sum[f] = 0.0f;
    for (int k = 0; k < p.top; ++k) {
        const int slot = row * p.top + k;
        const int expert = *static_cast<const volatile int32_t*>(p.chosen + slot);
        if (expert >= p.experts) continue;   // (the whole CTA: an identity expert)
        const float weight = p.weigh_results ? __ldg(p.weight + slot) : 1.0f;
        __syncthreads();
        for (int c = threadIdx.x; c < p.ff; c += kStreamThreads) x[c] = act[static_cast<int64_t>(slot) * p.ff + c] * weight;
        __syncthreads();
        const W* w[F];
#pragma unroll
        for (int f = 0; f < F; ++f) w[f] = static_cast<const W*>(p.down) + (static_cast<int64_t>(expert) * p.in + min(f0 + f, p.in - 1)) * p.ff;
        if (f0 < p.in) dot_rows<W, VECTOR, F>(w, x, p.ff, lane, sum);
    }
    const float through = identity_weight(p, row) * (p.identity > 0 ? row_factor(p, row) : 1.0f);
#pragma unroll
    for (int f = 0; f < F; ++f) {
        float v = warp_sum(sum[f]);
        if (lane == f && f0 + f < p.in) {
            const int64_t at = static_cast<int64_t>(row) * p.in + f0 + f;
            if (through != 0.0f) v = fmaf(through, row_value(p, at), v);
            p.y[at] = p.residual ? p.residual[at] + v : v;
        }
    }
}

template <class W, bool VECTOR, int F> int launch_expert_up(const ExpertParams& p, float* act, size_t smem, cudaStream_t stream) {
    auto kernel = p.gated ? expert_up_kernel<W, VECTOR, F, true> : expert_up_kernel<W, VECTOR, F, false>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    const dim3 grid(static_cast<unsigned>(p.rows * p.top), static_cast<unsigned>((p.ff + kStreamWarps * F - 1) / (kStreamWarps * F)));
    return cuda_status(launch_dependent(kernel, grid, dim3(kStreamThreads), smem, stream, p, act), "expert_up_kernel launch");
}
template <class W, bool VECTOR, int F> int launch_expert_down(const ExpertParams& p, const float* act, size_t smem, cudaStream_t stream) {
    auto kernel = expert_down_kernel<W, VECTOR, F>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    const dim3 grid(static_cast<unsigned>(p.rows), static_cast<unsigned>((p.in + kStreamWarps * F - 1) / (kStreamWarps * F)));
    return cuda_status(launch_dependent(kernel, grid, dim3(kStreamThreads), smem, stream, p, act), "expert_down_kernel launch");
}
// Four features per warp, or one where that would leave SMs without a CTA.
template <class W, bool VECTOR> int launch_streamed(const ExpertParams& p, float* act, size_t up_smem, size_t down_smem, int sms, cudaStream_t stream) {
    const int64_t up = static_cast<int64_t>(p.rows) * p.top * ((p.ff + 31) / 32), down = static_cast<int64_t>(p.rows) * ((p.in + 31) / 32);
    const int status = up < 2 * sms ? launch_expert_up<W, VECTOR, 1>(p, act, up_smem, stream) : launch_expert_up<W, VECTOR, 4>(p, act, up_smem, stream);
    if (status != B200_OK) return status;
    return down < 2 * sms ? launch_expert_down<W, VECTOR, 1>(p, act, down_smem, stream) : launch_expert_down<W, VECTOR, 4>(p, act, down_smem, stream);
}

// ---- grouped --------------------------------------------------------------------------------------------------------
constexpr int kTile = 128;        // features per weight tile, rows of the products
constexpr int kBlockK = 64;
constexpr int kBox = 32;          // slots per activation box
constexpr int kBoxBytes = kBox * kBlockK * 2;
constexpr int kWeightBytes = kTile * kBlockK * 2;
constexpr int kTileStride = kTile + 4;
constexpr int kGroupedThreads = 192;
// SLOTS: slots of a row tile.  The products always have 128 rows; what a smaller tile leaves out of the stage goes to further stages,
// that is to more weights in flight, and the rows past its slots multiply whatever lies behind them in shared memory: results that
// nobody reads.
template <int SLOTS> struct GroupedShape {
    static constexpr int kPlaneBytes = SLOTS * kBlockK * 2;
    static constexpr int kStageBytes = 2 * kPlaneBytes + kWeightBytes;   // W, x_hi, x_lo of one K block
    static constexpr int kStages = SLOTS == 128 ? 3 : SLOTS == 64 ? 5 : 8;
    static constexpr int kTileBytes = SLOTS * kTileStride * 4;
    static constexpr int kTileAt = kStages * kStageBytes;
    static constexpr int kControlAt = kTileAt + kTileBytes;
    static constexpr int kSmem = kControlAt + 1024 + 2048;
    static_assert((kStages - 1) * kStageBytes + kWeightBytes + kPlaneBytes + kTile * kBlockK * 2 <= kControlAt + 2048, "rows past the slots must lie in shared memory");
};

struct Grouped {
    __nv_bfloat16 *x_hi, *x_lo;        // [slots, in] in order of their experts
    __nv_bfloat16 *act_hi, *act_lo;    // [slots, ff]
    float* y;                          // [slots, in]; shares the memory of x_hi and x_lo, which are read before it is written
    float* scale;                      // [slots]
    int32_t* place;                    // [slots] sorted place of slot (row, choice)
    int4* tiles;                       // (expert, first sorted slot, slots, -)
    int32_t* tile_count;
};

// Slots of a row tile: the smallest height that takes an average expert's slots.
int tile_slots(const ExpertParams& p) {
    const int average = p.rows * p.top / p.experts;
    return average <= 24 ? 32 : average <= 48 ? 64 : 128;
}
size_t round_up_256(size_t n) { return (n + 255) & ~static_cast<size_t>(255); }
int most_tiles(const ExpertParams& p) {
    const int slots = p.rows * p.top;
    return slots / tile_slots(p) + std::min(p.experts, slots);   // every expert has at most one tile that is not full
}
size_t grouped_layout(const ExpertParams& p, uint8_t* base, Grouped& g) {
    const size_t slots = static_cast<size_t>(p.rows) * p.top;
    size_t at = 0;
    auto take = [&](size_t bytes) { uint8_t* here = base + at; at += round_up_256(bytes); return here; };
    uint8_t* x = take(slots * p.in * 4);
    g.x_hi = reinterpret_cast<__nv_bfloat16*>(x);
    g.x_lo = g.x_hi + slots * p.in;
    g.y = reinterpret_cast<float*>(x);
    g.act_hi = reinterpret_cast<__nv_bfloat16*>(take(slots * p.ff * 2));
    g.act_lo = reinterpret_cast<__nv_bfloat16*>(take(slots * p.ff * 2));
    g.scale = reinterpret_cast<float*>(take(slots * 4));
    g.place = reinterpret_cast<int32_t*>(take(slots * 4));
    g.tiles = reinterpret_cast<int4*>(take(static_cast<size_t>(most_tiles(p)) * sizeof(int4)));
    g.tile_count = reinterpret_cast<int32_t*>(take(4));
    return at;
}

// One CTA per slot; CTA 0 also writes the list of row tiles.
__global__ void __launch_bounds__(256) expert_gather_kernel(const __grid_constant__ ExpertParams p, const __grid_constant__ Grouped g, const int32_t* rank,
                                                            const int32_t* counts, const int height) {
    extern __shared__ int32_t copy[];   // [experts]
    __shared__ int32_t before;
    grid_dependency_wait();
    grid_launch_dependents();
    const int slot = blockIdx.x, expert = __ldg(p.chosen + slot);
    const bool sorted = expert < p.experts;   // not an identity expert
    if (sorted && threadIdx.x < 32) {
        int total = 0;
        for (int e = threadIdx.x; e < expert; e += 32) total += counts[e];
        total = __reduce_add_sync(0xffffffffu, total);
        if (threadIdx.x == 0) before = total;
    }
    if (slot == 0)
        for (int e = threadIdx.x; e < p.experts; e += blockDim.x) copy[e] = counts[e];
    __syncthreads();
    if (sorted) {
        const int to = before + rank[slot];
        const int64_t from_at = static_cast<int64_t>(slot / p.top) * p.in, to_at = static_cast<int64_t>(to) * p.in;
        for (int c = threadIdx.x * 8; c < p.in; c += blockDim.x * 8) {
            *reinterpret_cast<uint4*>(g.x_hi + to_at + c) = *reinterpret_cast<const uint4*>(p.x_hi + from_at + c);
            *reinterpret_cast<uint4*>(g.x_lo + to_at + c) = *reinterpret_cast<const uint4*>(p.x_lo + from_at + c);
        }
        if (threadIdx.x == 0) {
            g.scale[to] = slot_scale(p, slot);
            g.place[slot] = to;
        }
    }
    if (slot == 0) {
        for (int e = threadIdx.x; e < p.experts; e += blockDim.x) {
            int tile = 0, row = 0;
            for (int i = 0; i < e; ++i) { tile += (copy[i] + height - 1) / height; row += copy[i]; }
            for (int left = copy[e]; left > 0; left -= height, row += height) g.tiles[tile++] = make_int4(e, row, min(left, height), 0);
            if (e == p.experts - 1) *g.tile_count = tile;
        }
    }
}

struct ExpertGemm {
    LinearParams base;          // rows = slots, in, out (features of one expert), results
    const int4* tiles;
    const int32_t* tile_count;
    const float* scale;         // [slots] or NULL
    int32_t* status;
    bool listed;                // the list is older than the kernel before: the first weights may be asked for while that one runs
};

// Order of the tiles: bands of kBand row tiles, inside a band feature tile after feature tile.  What the CTAs work on at a time - a
// band's rows and its few experts' weights - then stays in L2 until it is finished with.
constexpr int kBand = 16;
__device__ __forceinline__ void tile_place(int t, int row_tiles, int feature_tiles, int& row_tile, int& feature_tile) {
    const int band = t / (kBand * feature_tiles), inside = t - band * kBand * feature_tiles, height = min(kBand, row_tiles - band * kBand);
    feature_tile = inside / height;
    row_tile = band * kBand + inside - feature_tile * height;
}

template <int EPI, int SLOTS>
__global__ void __launch_bounds__(kGroupedThreads, 1) expert_gemm_kernel(const __grid_constant__ CUtensorMap map_hi, const __grid_constant__ CUtensorMap map_lo,
                                                                         const __grid_constant__ CUtensorMap map_w, const __grid_constant__ ExpertGemm gp) {
    using S = GroupedShape<SLOTS>;
    constexpr int kStages = S::kStages, kStageBytes = S::kStageBytes;
    const LinearParams& p = gp.base;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
    float* tile = reinterpret_cast<float*>(smem + S::kTileAt);
    uint8_t* control = smem + S::kControlAt;
    uint64_t* full = reinterpret_cast<uint64_t*>(control);
    uint64_t* empty = full + kStages;
    uint64_t* acc_full = empty + kStages;    // [2]
    uint64_t* acc_empty = acc_full + 2;      // [2]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile int* alive_flag = reinterpret_cast<volatile int*>(control + 256);
    float* row_scale = reinterpret_cast<float*>(control + 512);
    constexpr uint32_t kInstruction = mma_instruction_bf16(kTile, kTile);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int k_blocks = (p.in + kBlockK - 1) / kBlockK;
    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; ++s) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        for (int b = 0; b < 2; ++b) {
            mbar_init(&acc_full[b], 1);
            mbar_init(&acc_empty[b], 4);
        }
        *alive_flag = 1;
        mbar_fence_init();
        tma_prefetch_descriptor(&map_hi);
        tma_prefetch_descriptor(&map_lo);
        tma_prefetch_descriptor(&map_w);
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, 2 * kTile);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;

    const int k_blocks_ahead = gp.listed && warp == 0 ? min(k_blocks, kStages) : 0;   // K blocks of the first tile whose weights are on their way
    if (k_blocks_ahead > 0) {
        const int count = *static_cast<const volatile int32_t*>(gp.tile_count), width = (p.out + kTile - 1) / kTile;
        if (static_cast<int>(blockIdx.x) < count * width) {
            int row_tile, feature_tile;
            tile_place(blockIdx.x, count, width, row_tile, feature_tile);
            const int4 group = *reinterpret_cast<const int4*>(gp.tiles + row_tile);
            const int boxes = (group.z + kBox - 1) / kBox;
            if (elect_one()) {
                for (int i = 0; i < k_blocks_ahead; ++i) {
                    mbar_expect_tx(&full[i], static_cast<uint32_t>(kWeightBytes + 2 * boxes * kBoxBytes));
                    tma_load_2d(smem + i * kStageBytes, &map_w, i * kBlockK, group.x * p.out + feature_tile * kTile, &full[i]);
                }
            }
            __syncwarp();
        }
    }
    grid_dependency_wait();
    grid_launch_dependents();
    const int row_tiles = *gp.tile_count, feature_tiles = (p.out + kTile - 1) / kTile, tiles = row_tiles * feature_tiles;
    const int my_tiles = (tiles - static_cast<int>(blockIdx.x) + static_cast<int>(gridDim.x) - 1) / static_cast<int>(gridDim.x);

    if (warp == 0) {
        int it = 0;   // K blocks issued so far: the ring does not restart between tiles
        bool alive = true;
        for (int j = 0; j < my_tiles && alive; ++j) {
            const int t = blockIdx.x + j * gridDim.x;
            int row_tile, feature_tile;
            tile_place(t, row_tiles, feature_tiles, row_tile, feature_tile);
            const int4 group = __ldg(gp.tiles + row_tile);
            const int boxes = (group.z + kBox - 1) / kBox, weight_row = group.x * p.out + feature_tile * kTile;
            for (int i = 0; i < k_blocks; ++i, ++it) {
                const int s = it % kStages;
                if (!mbar_wait(&empty[s], ((it / kStages) & 1) ^ 1)) {
                    if (lane == 0) atomicExch(gp.status, B200_DEVICE_TIMEOUT);
                    alive = false;
                    break;
                }
                if (elect_one()) {
                    uint8_t* stage = smem + s * kStageBytes;
                    if (it >= k_blocks_ahead) {
                        mbar_expect_tx(&full[s], static_cast<uint32_t>(kWeightBytes + 2 * boxes * kBoxBytes));
                        tma_load_2d(stage, &map_w, i * kBlockK, weight_row, &full[s]);
                    }
                    for (int b = 0; b < boxes; ++b) {
                        tma_load_2d(stage + kWeightBytes + b * kBoxBytes, &map_hi, i * kBlockK, group.y + b * kBox, &full[s]);
                        tma_load_2d(stage + kWeightBytes + S::kPlaneBytes + b * kBoxBytes, &map_lo, i * kBlockK, group.y + b * kBox, &full[s]);
                    }
                }
                __syncwarp();
            }
        }
    } else if (warp == 1) {
        int it = 0;
        bool alive = true;
        for (int j = 0; j < my_tiles && alive; ++j) {
            const int buffer = j & 1;
            // the epilogue of the tile that used this buffer two tiles ago must have read it (passes at once for j < 2)
            if (!mbar_wait(&acc_empty[buffer], ((j >> 1) & 1) ^ 1)) {
                if (lane == 0) atomicExch(gp.status, B200_DEVICE_TIMEOUT);
                break;
            }
            tc_fence_after_sync();
            const uint32_t accumulator = tmem_base + static_cast<uint32_t>(buffer * kTile);
            for (int i = 0; i < k_blocks; ++i, ++it) {
                const int s = it % kStages;
                if (!mbar_wait(&full[s], (it / kStages) & 1)) {
                    if (lane == 0) atomicExch(gp.status, B200_DEVICE_TIMEOUT);
                    alive = false;
                    break;
                }
                tc_fence_after_sync();
                if (elect_one()) {
                    const uint32_t stage = smem_u32(smem + s * kStageBytes);
                    const uint64_t w = operand_descriptor(stage), hi = operand_descriptor(stage + kWeightBytes);
                    const uint64_t lo = operand_descriptor(stage + kWeightBytes + S::kPlaneBytes);
#pragma unroll
                    for (int k = 0; k < kBlockK / 16; ++k) {
                        tc_mma_bf16(accumulator, hi + 2 * k, w + 2 * k, kInstruction, (i | k) != 0);
                        tc_mma_bf16(accumulator, lo + 2 * k, w + 2 * k, kInstruction, 1);
                    }
                    tc_commit(&empty[s]);
                    if (i == k_blocks - 1) tc_commit(&acc_full[buffer]);
                }
                __syncwarp();
            }
        }
    } else {
        // ---- epilogue warps 2-5: TMEM lanes 32 * (warp % 4) .. + 31; named barrier 2 joins the four warps ----
        const int quarter = warp & 3;
        const int tile_row = quarter * 32 + lane;
        const uint32_t own_tile[8] = {smem_u32(tile), 0u, 0u, 0u, 0u, 0u, 0u, 0u};
        for (int j = 0; j < my_tiles; ++j) {
            const int t = blockIdx.x + j * gridDim.x;
            int row_tile, feature_tile;
            tile_place(t, row_tiles, feature_tiles, row_tile, feature_tile);
            const int4 group = __ldg(gp.tiles + row_tile);
            const int n0 = feature_tile * kTile, buffer = j & 1;
            row_scale[tile_row] = gp.scale && tile_row < group.z ? __ldg(gp.scale + group.y + tile_row) : 1.0f;
            const bool ready = mbar_wait_relaxed(&acc_full[buffer], (j >> 1) & 1);
            if (!ready && lane == 0) { atomicExch(gp.status, B200_DEVICE_TIMEOUT); *alive_flag = 0; }
            tc_fence_after_sync();
            if (ready && quarter * 32 < group.z) {   // (so tile_row < SLOTS) lanes past the group's slots hold no results
#pragma unroll 1
                for (int c = 0; c < kTile / 32; ++c) {
                    uint32_t r[32];
                    tmem_load_32(tmem_base + (static_cast<uint32_t>(quarter * 32) << 16) + static_cast<uint32_t>(buffer * kTile + c * 32), r);
                    float4* out4 = reinterpret_cast<float4*>(tile + tile_row * kTileStride + c * 32);
#pragma unroll
                    for (int q = 0; q < 8; ++q)
                        out4[q] = make_float4(__uint_as_float(r[4 * q]), __uint_as_float(r[4 * q + 1]), __uint_as_float(r[4 * q + 2]),
                                              __uint_as_float(r[4 * q + 3]));
                }
            }
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[buffer]);
            asm volatile("bar.sync 2, 128;" ::: "memory");    // the tile and the row scales are in shared memory
            if (*alive_flag == 0) break;                       // same decision in all four warps
            finish_rows<EPI, kTile>(p, tile, own_tile, 1, row_scale, group.y, n0, feature_tile, 0, group.z, quarter, 4, lane, true);
            asm volatile("bar.sync 2, 128;" ::: "memory");    // the next tile may overwrite the shared-memory tile
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem_base, 2 * kTile);
    }
}

// One CTA per row: y = residual + the row's results in the order of its choices.  FINISH: the sum goes through the norm behind the mixture.
template <bool FINISH>
__global__ void __launch_bounds__(256) expert_combine_kernel(const __grid_constant__ ExpertParams p, const float* results, const int32_t* place) {
    __shared__ float scratch[FINISH ? 32 : 1];
    grid_dependency_wait();
    grid_launch_dependents();
    const int row = blockIdx.x;
    const int64_t at = static_cast<int64_t>(row) * p.in;
    const float through = p.identity > 0 ? identity_weight(p, row) * row_factor(p, row) : 0.0f;
    auto total = [&](int c, float4 sum) {
        for (int k = 0; k < p.top; ++k) {
            const int slot = row * p.top + k;
            if (p.identity > 0 && __ldg(p.chosen + slot) >= p.experts) continue;
            const float4 v = __ldcs(reinterpret_cast<const float4*>(results + static_cast<int64_t>(__ldg(place + slot)) * p.in + c));
            const float w = p.weigh_results ? __ldg(p.weight + slot) : 1.0f;
            sum.x = fmaf(v.x, w, sum.x); sum.y = fmaf(v.y, w, sum.y); sum.z = fmaf(v.z, w, sum.z); sum.w = fmaf(v.w, w, sum.w);
        }
        if (through != 0.0f) {
            const uint2 hi = *reinterpret_cast<const uint2*>(p.x_hi + at + c), lo = *reinterpret_cast<const uint2*>(p.x_lo + at + c);
            sum.x = fmaf(through, bf16_lo(hi.x) + bf16_lo(lo.x), sum.x);
            sum.y = fmaf(through, bf16_hi(hi.x) + bf16_hi(lo.x), sum.y);
            sum.z = fmaf(through, bf16_lo(hi.y) + bf16_lo(lo.y), sum.z);
            sum.w = fmaf(through, bf16_hi(hi.y) + bf16_hi(lo.y), sum.w);
        }
        return sum;
    };
    if constexpr (FINISH) {
        finish_sandwich<4, true>(p.after, row, p.in, [&](int c) {
            const float4 v = total(c, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
            return Lanes<4>{{v.x, v.y, v.z, v.w}};
        }, scratch);
    } else {
        for (int c = threadIdx.x * 4; c < p.in; c += blockDim.x * 4) {
            const float4 sum = p.residual ? *reinterpret_cast<const float4*>(p.residual + at + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            *reinterpret_cast<float4*>(p.y + at + c) = total(c, sum);
        }
    }
}

int encode_plane(CUtensorMap* map, const void* base, int64_t rows, int columns, int box_rows) {
    encode_tiled_fn encode = tensor_map_encoder();
    if (!encode) { set_error("cuTensorMapEncodeTiled is not available from this driver"); return B200_NO_DEVICE; }
    const cuuint64_t dims[2] = {static_cast<cuuint64_t>(columns), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[1] = {static_cast<cuuint64_t>(columns) * 2};
    const cuuint32_t box[2] = {kBlockK, static_cast<cuuint32_t>(box_rows)};
    const cuuint32_t element_strides[2] = {1, 1};
    const CUresult result = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, element_strides,
                                   CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (result != CUDA_SUCCESS) { set_error("cuTensorMapEncodeTiled(experts) failed with %d", static_cast<int>(result)); return B200_BAD_ARGUMENT; }
    return B200_OK;
}

template <int EPI, int SLOTS>
int launch_expert_tiles(const CUtensorMap& hi, const CUtensorMap& lo, const CUtensorMap& w, const ExpertGemm& gp, int ctas, cudaStream_t stream) {
    auto kernel = expert_gemm_kernel<EPI, SLOTS>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, GroupedShape<SLOTS>::kSmem));
    return cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(ctas)), dim3(kGroupedThreads), GroupedShape<SLOTS>::kSmem, stream, hi, lo, w, gp),
                       "expert_gemm_kernel launch");
}

template <int EPI>
int launch_expert_gemm(const ExpertParams& e, const Grouped& g, const __nv_bfloat16* hi, const __nv_bfloat16* lo, const void* weight, int in, int out,
                       ExpertGemm gp, int sms, cudaStream_t stream) {
    alignas(64) CUtensorMap map_hi, map_lo, map_w;
    const int slots = e.rows * e.top;
    int status = encode_plane(&map_hi, hi, slots, in, kBox);
    if (status == B200_OK) status = encode_plane(&map_lo, lo, slots, in, kBox);
    if (status == B200_OK) status = encode_plane(&map_w, weight, static_cast<int64_t>(e.experts) * out, in, kTile);
    if (status != B200_OK) return status;
    gp.base.rows = slots; gp.base.in = in; gp.base.out = out;
    gp.tiles = g.tiles; gp.tile_count = g.tile_count;
    const int ctas = static_cast<int>(std::min<int64_t>(static_cast<int64_t>(most_tiles(e)) * ((out + kTile - 1) / kTile), sms));
    switch (tile_slots(e)) {
    case 32: return launch_expert_tiles<EPI, 32>(map_hi, map_lo, map_w, gp, ctas, stream);
    case 64: return launch_expert_tiles<EPI, 64>(map_hi, map_lo, map_w, gp, ctas, stream);
    default: return launch_expert_tiles<EPI, 128>(map_hi, map_lo, map_w, gp, ctas, stream);
    }
}

// Slots up to which every slot streams its expert on its own.
constexpr int kStreamedSlots = 16;

bool takes_grouped(const b200_experts* a, const ExpertParams& p) {
    return a->weight_dtype == B200_BF16 && p.x_hi && p.x_lo && p.in % 8 == 0 && p.ff % 8 == 0
        && ((reinterpret_cast<uintptr_t>(p.x_hi) | reinterpret_cast<uintptr_t>(p.x_lo) | reinterpret_cast<uintptr_t>(p.up) | reinterpret_cast<uintptr_t>(p.down)
             | reinterpret_cast<uintptr_t>(p.residual) | reinterpret_cast<uintptr_t>(p.y)) & 15) == 0
        && (!p.finishes || sandwich_takes_quads(p.after, p.in));
}

constexpr int kRouteWarps = 8;
__global__ void __launch_bounds__(kRouteWarps * 32) route_rows_kernel(const float* logits, const int rows, const int64_t stride, const __grid_constant__ Route route) {
    extern __shared__ float copies[];   // [warps][experts]
    grid_dependency_wait();
    grid_launch_dependents();
    const int warp = threadIdx.x >> 5, row = blockIdx.x * kRouteWarps + warp;
    if (row < rows) choose_experts(route, row, logits + row * stride, copies + warp * route.experts, threadIdx.x & 31);
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int32_t b200_experts_takes_grouped(const b200_experts* args) {
    ExpertParams p;
    return expert_params(args, p) && takes_grouped(args, p) && p.rows * p.top > kStreamedSlots;
}

extern "C" size_t b200_experts_grouped_bytes(const b200_experts* args) {
    ExpertParams p;
    Grouped g;
    return expert_params(args, p) ? grouped_layout(p, nullptr, g) : 0;
}

extern "C" int b200_experts_grouped(const b200_experts* args, const int32_t* rank, const int32_t* counts, void* scratch, size_t scratch_bytes, void* stream) {
    ExpertParams p;
    Grouped g;
    if (!expert_params(args, p)) return B200_BAD_ARGUMENT;
    if (!rank || !counts || !scratch || (reinterpret_cast<uintptr_t>(scratch) & 255) || scratch_bytes < grouped_layout(p, static_cast<uint8_t*>(scratch), g)) {
        set_error("b200_experts_grouped: bad workspace");
        return B200_BAD_ARGUMENT;
    }
    if (!takes_grouped(args, p)) { set_error("b200_experts_grouped: needs bf16 planes and widths that are multiples of 8"); return B200_UNSUPPORTED; }
    int device = 0;
    B200_CUDA(cudaGetDevice(&device));
    ExpertGemm gp{};
    gp.status = device_status_word(device);
    if (!gp.status) { set_error("the device status word could not be allocated"); return B200_NO_DEVICE; }
    const int sms = sm_count(device), slots = p.rows * p.top;
    cudaStream_t s = as_stream(stream);
    int status = cuda_status(launch_dependent(expert_gather_kernel, dim3(static_cast<unsigned>(slots)), dim3(256), static_cast<size_t>(p.experts) * 4, s, p, g, rank,
                                              counts, tile_slots(p)), "expert_gather_kernel launch");
    if (status != B200_OK) return status;
    ExpertGemm up = gp, down = gp;
    up.scale = g.scale;
    up.base.out_hi = g.act_hi; up.base.out_lo = g.act_lo;
    up.base.out_stride = p.ff;
    status = p.gated ? launch_expert_gemm<B200_EPI_SWIGLU>(p, g, g.x_hi, g.x_lo, p.up, p.in, 2 * p.ff, up, sms, s)
                     : launch_expert_gemm<B200_EPI_GELU>(p, g, g.x_hi, g.x_lo, p.up, p.in, p.ff, up, sms, s);
    if (status != B200_OK) return status;
    down.base.y = g.y;
    down.listed = true;
    status = launch_expert_gemm<B200_EPI_STORE>(p, g, g.act_hi, g.act_lo, p.down, p.ff, p.in, down, sms, s);
    if (status != B200_OK) return status;
    return cuda_status(launch_dependent(p.finishes ? expert_combine_kernel<true> : expert_combine_kernel<false>, dim3(static_cast<unsigned>(p.rows)), dim3(256), 0, s, p, static_cast<const float*>(g.y),
                                        static_cast<const int32_t*>(g.place)), "expert_combine_kernel launch");
}

extern "C" int b200_experts_streamed(const b200_experts* args, float* act, void* stream) {
    ExpertParams p;
    if (args && args->after) { set_error("b200_experts_streamed: the norm behind the mixture belongs to the grouped form"); return B200_BAD_ARGUMENT; }
    if (!expert_params(args, p) || !act) { if (!act) set_error("b200_experts_streamed: no workspace"); return B200_BAD_ARGUMENT; }
    const size_t up_smem = (static_cast<size_t>(p.in) * 4 + 15) & ~15ull, down_smem = (static_cast<size_t>(p.ff) * 4 + 15) & ~15ull;
    if (up_smem > 220 * 1024 || down_smem > 220 * 1024 || p.ff > 65535 * kStreamWarps || p.in > 65535 * kStreamWarps) {
        set_error("b200_experts_streamed: widths %d and %d are too large", p.in, p.ff);
        return B200_UNSUPPORTED;
    }
    const bool bf16 = args->weight_dtype == B200_BF16;
    const int per = bf16 ? 8 : 4;
    const bool vector = p.in % per == 0 && p.ff % per == 0 && ((reinterpret_cast<uintptr_t>(p.up) | reinterpret_cast<uintptr_t>(p.down)) & 15) == 0;
    int device = 0;
    B200_CUDA(cudaGetDevice(&device));
    const int sms = sm_count(device);
    cudaStream_t s = as_stream(stream);
    if (bf16) return vector ? launch_streamed<__nv_bfloat16, true>(p, act, up_smem, down_smem, sms, s) : launch_streamed<__nv_bfloat16, false>(p, act, up_smem, down_smem, sms, s);
    return vector ? launch_streamed<float, true>(p, act, up_smem, down_smem, sms, s) : launch_streamed<float, false>(p, act, up_smem, down_smem, sms, s);
}

extern "C" int b200_route_rows(const float* logits, int64_t rows, int64_t stride, const b200_route* route, void* stream) {
    Route r;
    if (!logits || rows < 0 || rows > INT32_MAX || !route || !route_view(route, r) || stride < r.experts || rows * r.top > INT32_MAX) {
        set_error("b200_route_rows: bad pointer or size");
        return B200_BAD_ARGUMENT;
    }
    if (rows == 0) return B200_OK;
    return cuda_status(launch_dependent(route_rows_kernel, dim3(static_cast<unsigned>((rows + kRouteWarps - 1) / kRouteWarps)), dim3(kRouteWarps * 32),
                                        static_cast<size_t>(kRouteWarps) * r.experts * 4, as_stream(stream), logits, static_cast<int>(rows), stride, r),
                       "route_rows_kernel launch");
}
