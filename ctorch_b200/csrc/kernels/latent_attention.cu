// Latent attention over a paged cache of latents: per token one latent vector (kv_rank values) and one rotated key part shared by
// all heads.  The key and value up-projections are absorbed: a query is taken through its head's key up-projection once
// (b200_latent_query), attends to the latents themselves, and the weighted latent goes through the value up-projection
// (b200_latent_value).  Every cached byte serves all heads as key and as value.
//
//   * latent_mma_kernel: bf16 caches.  Half pages arrive through a TMA ring as boxes of 32 tokens x 64 values (128-byte swizzle,
//     one copy for all of them, mbarrier completion); the consumer warps hold the queries as tensor-core fragments in registers, the query-key product split 4 ways over the
//     width and 4 or 2 ways over the keys of a page; the partial scores meet in shared memory, a warp finishes whole rows of the
//     online softmax in f32; then every warp multiplies the weights (as hi + lo planes) with its columns of the same page.
//     Decode: 16 rows (heads of one token), 16 warps.  Longer passes and wide head counts: 32 rows, 8 warps.
//   * latent_generic_kernel: f32 caches and odd sizes, f32 FMAs, one (row, head) per CTA.
#include "kv_cache.cuh"
#include "mma.cuh"
#include "rows.cuh"

#include <algorithm>

namespace b200 {
namespace {

struct LatentParams {
    int heads, dim, rot_dim, vdim, rank, q_rank, rot_dims, width;   // width = rank + rot_dim
    float scale, eps;
    const float *cosine, *sine;
    int positions;
    const float *q_norm, *kv_norm;
    KvView kv;
    int weight_dtype;
    const void *w_key, *w_value;
};

bool latent_params(const b200_latent_args* a, LatentParams& p, bool needs_cache) {
    if (!a || a->heads <= 0 || a->dim <= 0 || a->rot_dim < 0 || a->vdim <= 0 || a->kv_rank <= 0 || a->q_rank <= 0 || a->rot_dims < 0
        || (a->rot_dims & 1) || a->rot_dims > a->rot_dim || (a->rot_dims > 0 && (!a->cosine || !a->sine)) || !a->q_norm || !a->kv_norm
        || !a->w_key || !a->w_value || (a->weight_dtype != B200_F32 && a->weight_dtype != B200_BF16)) {
        set_error("latent attention: bad pointer or size");
        return false;
    }
    p = LatentParams{};
    p.heads = a->heads; p.dim = a->dim; p.rot_dim = a->rot_dim; p.vdim = a->vdim; p.rank = a->kv_rank; p.q_rank = a->q_rank;
    p.rot_dims = a->rot_dims; p.width = a->kv_rank + a->rot_dim;
    p.scale = a->scale; p.eps = static_cast<float>(a->eps);
    p.cosine = a->cosine; p.sine = a->sine; p.positions = a->positions; p.q_norm = a->q_norm; p.kv_norm = a->kv_norm;
    p.weight_dtype = a->weight_dtype; p.w_key = a->w_key; p.w_value = a->w_value;
    if (needs_cache) {
        if (!a->cache) { set_error("latent attention: no cache"); return false; }
        p.kv = kv_view(a->cache);
        if (p.kv.kv_heads != 1 || p.kv.head_dim != p.width) { set_error("latent attention: the cache has another width"); return false; }
    }
    return true;
}

// Entry i of a rotated part: interleaved pairs (2j, 2j + 1) turned by the angle of pair j at `position`; the rest passes.
__device__ __forceinline__ float rotated(const LatentParams& p, const float* part, int i, int position) {
    const float v = part[i];
    if (i >= p.rot_dims || static_cast<unsigned>(position) >= static_cast<unsigned>(p.positions)) return v;
    const int64_t at = static_cast<int64_t>(position) * (p.rot_dims >> 1) + (i >> 1);
    const float c = __ldg(p.cosine + at), s = __ldg(p.sine + at);
    return i & 1 ? __fadd_rn(__fmul_rn(v, c), __fmul_rn(part[i - 1], s)) : __fsub_rn(__fmul_rn(v, c), __fmul_rn(part[i + 1], s));
}

__device__ __forceinline__ void cache_store(const KvView& kv, int64_t at, float v) {
    if (kv.dtype == B200_BF16) static_cast<__nv_bfloat16*>(kv.pool[0])[at] = __float2bfloat16_rn(v);
    else static_cast<float*>(kv.pool[0])[at] = v;
}

// One CTA per row.
__global__ void __launch_bounds__(256) latent_prepare_kernel(const LatentParams p, const RowsView rows, const float* projected, int64_t stride,
                                                             float* q_latent, __nv_bfloat16* q_hi, __nv_bfloat16* q_lo) {
    __shared__ float scratch[32];
    grid_dependency_wait();
    grid_launch_dependents();
    const int row = blockIdx.x;
    const RowPlace place = row_place(rows, row);
    const float* query = projected + row * stride;
    const float* latent = query + p.q_rank;
    const float* key = latent + p.rank;
    float qs = 0.0f, ks = 0.0f;
    for (int c = threadIdx.x; c < p.q_rank; c += blockDim.x) qs = fmaf(query[c], query[c], qs);
    for (int c = threadIdx.x; c < p.rank; c += blockDim.x) ks = fmaf(latent[c], latent[c], ks);
    qs = block_sum(qs, scratch);
    ks = block_sum(ks, scratch);
    const float q_inverse = 1.0f / sqrtf(qs / static_cast<float>(p.q_rank) + p.eps);
    const float k_inverse = 1.0f / sqrtf(ks / static_cast<float>(p.rank) + p.eps);
    for (int c = threadIdx.x; c < p.q_rank; c += blockDim.x)
        store_forms(query[c] * q_inverse * p.q_norm[c], static_cast<int64_t>(row) * p.q_rank + c, q_latent, q_hi, q_lo);
    if (place.position >= p.kv.pages_per_seq * p.kv.page_size) return;   // the host refuses passes that do not fit
    const int64_t at = kv_offset(p.kv, place.slot, place.position, 0);
    for (int c = threadIdx.x; c < p.rank; c += blockDim.x) cache_store(p.kv, at + c, latent[c] * k_inverse * p.kv_norm[c]);
    for (int c = threadIdx.x; c < p.rot_dim; c += blockDim.x) cache_store(p.kv, at + p.rank + c, rotated(p, key, c, place.position));
}

// ---- per-head projections ---------------------------------------------------------------------------------------
// y[row, head, o] = sum_k x[row, head, k] w[head][o][k] for two callers: the absorbed query (results stored at the head's slice of
// the wide query, plus its rotated part) and the value up-projection (results gated, stored as f32 or planes).
struct HeadLinear {
    LatentParams latent;
    RowsView rows;           // query form only
    const float* x;
    int64_t x_row, x_head;   // strides of x
    int row_count, in, out;
    const void* w;
    bool query;
    float* y;                // query form: [rows, heads, width]
    const float* gate;       // value form
    int64_t gate_stride;
    __nv_bfloat16 *out_hi, *out_lo;
};

__device__ __forceinline__ void head_result(const HeadLinear& h, int row, int head, int o, float v) {
    if (h.query) {
        h.y[(static_cast<int64_t>(row) * h.latent.heads + head) * h.latent.width + o] = v;
    } else {
        const int64_t column = static_cast<int64_t>(head) * h.out + o;
        const float g = h.gate[row * h.gate_stride + column];
        store_forms(v * (1.0f / (1.0f + expf(-g))), row * static_cast<int64_t>(h.latent.heads) * h.out + column, h.y, h.out_hi, h.out_lo);
    }
}
__device__ __forceinline__ void head_rotated(const HeadLinear& h, int row, int head, int i, int position) {
    const LatentParams& p = h.latent;
    const float* part = h.x + row * h.x_row + head * h.x_head + p.dim;
    h.y[(static_cast<int64_t>(row) * p.heads + head) * p.width + p.rank + i] = rotated(p, part, i, position);
}

// One warp per output; grid (output blocks, rows, heads).
template <class W> __global__ void __launch_bounds__(256) head_linear_generic_kernel(const __grid_constant__ HeadLinear h) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.y, head = blockIdx.z;
    const float* x = h.x + row * h.x_row + head * h.x_head;
    for (int o = blockIdx.x * 64 + warp; o < min(h.out, static_cast<int>(blockIdx.x + 1) * 64); o += 8) {
        const W* w = static_cast<const W*>(h.w) + (static_cast<int64_t>(head) * h.out + o) * h.in;
        float acc = 0.0f;
        for (int k = lane; k < h.in; k += 32) acc = fmaf(x[k], load_as_f32(w, k), acc);
        acc = warp_sum(acc);
        if (lane == 0) head_result(h, row, head, o, acc);
    }
    if (h.query && blockIdx.x == 0)
        for (int i = threadIdx.x; i < h.latent.rot_dim; i += blockDim.x) head_rotated(h, row, head, i, row_place(h.rows, row).position);
}

// bf16 weights on the tensor cores; the f32 inputs are split into planes while they are staged.  WM x WN warps, each MI x 16 rows by
// NI x 8 outputs; KC input columns at a time, double-buffered, the next chunk's rows fetched into registers under the products.
template <int WM, int WN, int MI, int NI, int KC> struct HeadTile {
    static constexpr int kThreads = WM * WN * 32, kM = WM * MI * 16, kN = WN * NI * 8, kPitch = KC + 8;
    static constexpr int kSmem = 2 * (2 * kM + kN) * kPitch * 2;
    static constexpr int kQuads = kM * KC / 4 / kThreads;
};

template <int WM, int WN, int MI, int NI, int KC, bool QUERY>
__global__ void __launch_bounds__(WM * WN * 32, WM * WN == 8 ? 2 : 1) head_linear_mma_kernel(const __grid_constant__ HeadLinear h) {
    using Tile = HeadTile<WM, WN, MI, NI, KC>;
    constexpr int kPitch = Tile::kPitch;
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ int positions[Tile::kM];
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(smem);            // [2 buffers][2 planes][kM][pitch]
    __nv_bfloat16* ws = xs + 4 * Tile::kM * kPitch;                        // [2 buffers][kN][pitch]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int o0 = blockIdx.x * Tile::kN, row0 = blockIdx.y * Tile::kM, head = blockIdx.z;
    const __nv_bfloat16* weight = static_cast<const __nv_bfloat16*>(h.w) + static_cast<int64_t>(head) * h.out * h.in;
    auto stage_weights = [&](int chunk) {
        __nv_bfloat16* dst = ws + (chunk & 1) * Tile::kN * kPitch;
        for (int i = threadIdx.x; i < Tile::kN * (KC / 8); i += Tile::kThreads) {
            const int o = i / (KC / 8), c = (i % (KC / 8)) * 8, k = chunk * KC + c;
            const bool live = o0 + o < h.out && k < h.in;
            copy_async_16(smem_u32(dst + o * kPitch + c), live ? weight + static_cast<int64_t>(o0 + o) * h.in + k : weight, live);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float4 ahead[Tile::kQuads];
    auto fetch_rows = [&](int chunk) {
#pragma unroll
        for (int j = 0; j < Tile::kQuads; ++j) {
            const int i = threadIdx.x + j * Tile::kThreads, r = i / (KC / 4), k = chunk * KC + (i % (KC / 4)) * 4;
            ahead[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (row0 + r < h.row_count && k < h.in)
                ahead[j] = *reinterpret_cast<const float4*>(h.x + (row0 + r) * h.x_row + head * h.x_head + k);
        }
    };
    auto put_rows = [&](int chunk) {
        __nv_bfloat16* hi = xs + (chunk & 1) * 2 * Tile::kM * kPitch;
        __nv_bfloat16* lo = hi + Tile::kM * kPitch;
#pragma unroll
        for (int j = 0; j < Tile::kQuads; ++j) {
            const int i = threadIdx.x + j * Tile::kThreads, r = i / (KC / 4), c = (i % (KC / 4)) * 4;
            uint32_t h0, l0, h1, l1;
            pack_planes(ahead[j].x, ahead[j].y, h0, l0);
            pack_planes(ahead[j].z, ahead[j].w, h1, l1);
            *reinterpret_cast<uint2*>(hi + r * kPitch + c) = make_uint2(h0, h1);
            *reinterpret_cast<uint2*>(lo + r * kPitch + c) = make_uint2(l0, l1);
        }
    };
    float acc[MI][NI][4];
#pragma unroll
    for (int m = 0; m < MI; ++m)
#pragma unroll
        for (int n = 0; n < NI; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.0f;

    const int chunks = (h.in + KC - 1) / KC;
    const int m0 = (warp / WN) * MI * 16, n0 = (warp % WN) * NI * 8;
    stage_weights(0);          // weights are constants: requested before the producer of x is waited for
    grid_dependency_wait();
    grid_launch_dependents();
    fetch_rows(0);
    if constexpr (QUERY) {
        if (threadIdx.x < Tile::kM && row0 + static_cast<int>(threadIdx.x) < h.row_count)
            positions[threadIdx.x] = row_place(h.rows, row0 + threadIdx.x).position;
    }
    put_rows(0);
    for (int chunk = 0; chunk < chunks; ++chunk) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (chunk + 1 < chunks) { stage_weights(chunk + 1); fetch_rows(chunk + 1); }
        const __nv_bfloat16* hi = xs + (chunk & 1) * 2 * Tile::kM * kPitch;
        const uint32_t a_hi = smem_u32(hi + (m0 + (lane & 15)) * kPitch + (lane >> 4) * 8);
        const uint32_t a_lo = a_hi + Tile::kM * kPitch * 2;
        const uint32_t b = smem_u32(ws + (chunk & 1) * Tile::kN * kPitch + (n0 + (lane >> 4) * 8 + (lane & 7)) * kPitch + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int k = 0; k < KC / 16; ++k) {
            uint32_t a[2][MI][4], w[NI / 2][4];
#pragma unroll
            for (int m = 0; m < MI; ++m) {
                ldsm_x4(a[0][m], a_hi + m * 16 * kPitch * 2 + k * 32);
                ldsm_x4(a[1][m], a_lo + m * 16 * kPitch * 2 + k * 32);
            }
#pragma unroll
            for (int n = 0; n < NI / 2; ++n) ldsm_x4(w[n], b + n * 16 * kPitch * 2 + k * 32);
#pragma unroll
            for (int plane = 0; plane < 2; ++plane)
#pragma unroll
                for (int m = 0; m < MI; ++m)
#pragma unroll
                    for (int n = 0; n < NI; ++n) mma_16816(acc[m][n], a[plane][m], w[n >> 1][(n & 1) * 2], w[n >> 1][(n & 1) * 2 + 1]);
        }
        if (chunk + 1 < chunks) put_rows(chunk + 1);
    }
    const LatentParams& p = h.latent;
#pragma unroll
    for (int m = 0; m < MI; ++m)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int row = row0 + m0 + m * 16 + (lane >> 2) + i * 8, o = o0 + n0 + (lane & 3) * 2;
            if (row >= h.row_count) continue;
            if constexpr (QUERY) {
                float* to = h.y + (static_cast<int64_t>(row) * p.heads + head) * p.width + o;
#pragma unroll
                for (int n = 0; n < NI; ++n)
                    if (o + n * 8 < h.out) *reinterpret_cast<float2*>(to + n * 8) = make_float2(acc[m][n][2 * i], acc[m][n][2 * i + 1]);
            } else {
                const int64_t column = static_cast<int64_t>(head) * h.out + o, at = static_cast<int64_t>(row) * p.heads * h.out + column;
                const float* gate = h.gate + row * h.gate_stride + column;
                float2 g[NI];   // all gates of the row before the first store
#pragma unroll
                for (int n = 0; n < NI; ++n) {
                    g[n] = make_float2(0.0f, 0.0f);
                    if (o + n * 8 < h.out) g[n] = make_float2(__ldg(gate + n * 8), __ldg(gate + n * 8 + 1));
                }
#pragma unroll
                for (int n = 0; n < NI; ++n) {
                    if (o + n * 8 >= h.out) continue;
                    const float v0 = acc[m][n][2 * i] * (1.0f / (1.0f + expf(-g[n].x))), v1 = acc[m][n][2 * i + 1] * (1.0f / (1.0f + expf(-g[n].y)));
                    if (h.y) *reinterpret_cast<float2*>(h.y + at + n * 8) = make_float2(v0, v1);
                    if (h.out_hi) {
                        uint32_t hi, lo;
                        pack_planes(v0, v1, hi, lo);
                        *reinterpret_cast<uint32_t*>(h.out_hi + at + n * 8) = hi;
                        if (h.out_lo) *reinterpret_cast<uint32_t*>(h.out_lo + at + n * 8) = lo;
                    }
                }
            }
        }
    if constexpr (QUERY) {   // the output tiles of a head share the rows' rotated parts, a pair of values at a time
        const int pairs = p.rot_dim >> 1, live = min(Tile::kM, h.row_count - row0);
#pragma unroll 4
        for (int e = threadIdx.x + blockIdx.x * Tile::kThreads; e < live * pairs; e += gridDim.x * Tile::kThreads) {
            const int r = e / pairs, i = (e - r * pairs) * 2, position = positions[r];
            const float2 v = *reinterpret_cast<const float2*>(h.x + (row0 + r) * h.x_row + head * h.x_head + p.dim + i);
            float2 turned = v;
            if (i < p.rot_dims && static_cast<unsigned>(position) < static_cast<unsigned>(p.positions)) {
                const int64_t at = static_cast<int64_t>(position) * (p.rot_dims >> 1) + (i >> 1);
                const float c = __ldg(p.cosine + at), s = __ldg(p.sine + at);
                turned = make_float2(__fsub_rn(__fmul_rn(v.x, c), __fmul_rn(v.y, s)), __fadd_rn(__fmul_rn(v.y, c), __fmul_rn(v.x, s)));
            }
            *reinterpret_cast<float2*>(h.y + (static_cast<int64_t>(row0 + r) * p.heads + head) * p.width + p.rank + i) = turned;
        }
    }
}

template <int WM, int WN, int MI, int NI, int KC> int launch_head_mma(const HeadLinear& h, cudaStream_t stream) {
    using Tile = HeadTile<WM, WN, MI, NI, KC>;
    auto kernel = h.query ? head_linear_mma_kernel<WM, WN, MI, NI, KC, true> : head_linear_mma_kernel<WM, WN, MI, NI, KC, false>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, Tile::kSmem));
    const dim3 grid(static_cast<unsigned>((h.out + Tile::kN - 1) / Tile::kN), static_cast<unsigned>((h.row_count + Tile::kM - 1) / Tile::kM),
                    static_cast<unsigned>(h.latent.heads));
    return cuda_status(launch_dependent(kernel, grid, dim3(Tile::kThreads), Tile::kSmem, stream, h), "head_linear_mma_kernel launch");
}

int launch_head_linear(const HeadLinear& h, cudaStream_t stream) {
    const LatentParams& p = h.latent;
    if (h.row_count > 65535 || p.heads > 65535) { set_error("latent attention: at most 65535 rows and heads in one pass"); return B200_UNSUPPORTED; }
    const bool mma = p.weight_dtype == B200_BF16 && h.in % 8 == 0 && h.x_row % 4 == 0 && h.x_head % 4 == 0 && h.out % 2 == 0 && p.width % 2 == 0
        && p.rot_dim % 2 == 0
        && ((reinterpret_cast<uintptr_t>(h.x) | reinterpret_cast<uintptr_t>(h.w)) & 15) == 0 && (reinterpret_cast<uintptr_t>(h.y) & 7) == 0;
    if (!mma) {
        const dim3 grid(static_cast<unsigned>((h.out + 63) / 64), static_cast<unsigned>(h.row_count), static_cast<unsigned>(p.heads));
        return cuda_status(p.weight_dtype == B200_BF16 ? launch_dependent(head_linear_generic_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, h)
                                                       : launch_dependent(head_linear_generic_kernel<float>, grid, dim3(256), 0, stream, h),
                           "head_linear_generic_kernel launch");
    }
    if (h.row_count <= 256) return launch_head_mma<1, 4, 1, 2, 128>(h, stream);   // 16 rows x 64 outputs: CTAs for every SM
    return launch_head_mma<4, 2, 2, 8, 64>(h, stream);                            // 128 x 128: least traffic from L2
}

// ---- attention ----------------------------------------------------------------------------------------------------
struct LatentAttention {
    LatentParams latent;
    RowsView rows;
    const float* query;        // [rows, heads, width]
    float* out;                // [rows, heads, rank]
    int positions_per_item, head_chunk, head_chunks, splits;
    float *partial, *partial_ml;   // splits > 1: [rows, heads, splits, rank], [rows, heads, splits, 2]
    int stages;
    int32_t* status;
};

constexpr int kPage = 64;
constexpr int kScorePitch = 68, kWeightPitch = 72;

constexpr int kHalf = kLatentBoxRows;         // tokens of one ring stage: half a page
constexpr int kBoxBytes = kHalf * 64 * 2;    // one box: 32 tokens x 64 values
static_assert(2 * kHalf == kPage);
int latent_fixed_bytes(int m) { return 4 * m * kScorePitch * 4 + 2 * m * kWeightPitch * 2 + 4 * m * 4 + 256; }

// KS: 16-wide steps of the width per quarter; VT: 8-column tiles of the latent per warp; MT: 16-row tiles.
// MT = 1 (decode steps): 16 consumer warps and a producer warp, so that four warps per scheduler hide the products' latency and the
// copies run ahead on their own.  MT = 2 (longer passes, whose pages come from L2): 8 warps, which leaves 255 registers for the
// queries' and the result's fragments; warp 0 issues the copies as pages are finished with.
template <int MT> struct LatentShape {
    static constexpr int kWarps = MT == 1 ? 16 : 8, kConsumers = kWarps * 32;
    static constexpr bool kProducer = MT == 1;
    static constexpr int kThreads = kConsumers + (kProducer ? 32 : 0);
};
template <int THREADS> __device__ __forceinline__ void consumers_sync() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }

// Called by a whole warp.
__device__ __forceinline__ void latent_copy_half(const CUtensorMap* map, const int32_t* table, int half, uint8_t* stage, int boxes, uint64_t* full) {
    const int row = __ldg(table + (half >> 1)) * kPage + (half & 1) * kHalf;
    if (elect_one()) {
        mbar_expect_tx(full, static_cast<uint32_t>(boxes * kBoxBytes));
        tma_load_3d(stage, map, 0, row, 0, full);
    }
    __syncwarp();
}
// Byte offset of 16-byte chunk `chunk` (8 values) of a row inside a stage: boxes side by side, the chunk swizzled by its row.
__device__ __forceinline__ uint32_t stage_offset(int row, int chunk) {
    return static_cast<uint32_t>((chunk >> 3) * kBoxBytes + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}

template <int KS, int VT, int MT>
__global__ void __launch_bounds__(LatentShape<MT>::kThreads, 1) latent_mma_kernel(const __grid_constant__ LatentAttention a, const __grid_constant__ CUtensorMap map) {
    using Shape = LatentShape<MT>;
    constexpr int M = 16 * MT, kWarps = Shape::kWarps, kGroups = kWarps / 4, kKeyTiles = kPage / 8 / kGroups;   // key tiles per warp
    extern __shared__ __align__(16) uint8_t smem[];
    const LatentParams& p = a.latent;
    const int boxes = (p.width + 63) >> 6, stage_bytes = boxes * kBoxBytes;
    uint8_t* ring = smem + ((1024u - (smem_u32(smem) & 1023u)) & 1023u);             // swizzled boxes start on 1024-byte boundaries
    float* scores = reinterpret_cast<float*>(ring + a.stages * stage_bytes);         // [4][M][kScorePitch]
    __nv_bfloat16* weights = reinterpret_cast<__nv_bfloat16*>(scores + 4 * M * kScorePitch);   // [2 planes][M][kWeightPitch]
    float* shrink = reinterpret_cast<float*>(weights + 2 * M * kWeightPitch);       // [M] factor of the accumulators
    float* row_m = shrink + M;
    float* row_l = row_m + M;
    int* visible = reinterpret_cast<int*>(row_l + M);                               // [M] keys the row sees
    uint64_t* full = reinterpret_cast<uint64_t*>(visible + M);
    uint64_t* empty = full + 8;
    int* gave_up = reinterpret_cast<int*>(empty + 8);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = blockIdx.z % a.splits, chunk = blockIdx.z / a.splits, sequence = blockIdx.y;
    if (threadIdx.x == 0) {
        tma_prefetch_descriptor(&map);
        for (int s = 0; s < a.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], kWarps); }
        mbar_fence_init();
        *gave_up = 0;
    }
    grid_dependency_wait();
    grid_launch_dependents();
    const int first = __ldg(a.rows.first + sequence), count = __ldg(a.rows.first + sequence + 1) - first;
    const int slot = __ldg(a.rows.slot + sequence), length = a.rows.lengths[slot];
    // the items with the most keys start first
    const int offset = (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * a.positions_per_item;
    if (offset >= count) return;
    const int last = min(offset + a.positions_per_item, count);
    const int keys = length + last;
    const int pages = (keys + kPage - 1) / kPage, per_split = (pages + a.splits - 1) / a.splits;
    const int page0 = split * per_split, page1 = min(pages, page0 + per_split);
    if (threadIdx.x < M) {
        const int position = threadIdx.x / a.head_chunk, head = chunk * M + threadIdx.x % a.head_chunk;
        const bool live = position < a.positions_per_item && offset + position < last && head < p.heads;
        visible[threadIdx.x] = live ? length + offset + position + 1 : 0;
        shrink[threadIdx.x] = 1.0f;
    }
    __syncthreads();

    const int32_t* table = p.kv.page_table + static_cast<int64_t>(slot) * p.kv.pages_per_seq;
    if (Shape::kProducer && warp == kWarps) {
        int s = 0;
        uint32_t parity = 1;   // of the wait for a free stage; the first round does not wait
        for (int i = 0; i < 2 * (page1 - page0); ++i) {
            if (i >= a.stages && !mbar_wait(&empty[s], parity)) {
                if (lane == 0) atomicExch(a.status, B200_DEVICE_TIMEOUT);
                break;
            }
            latent_copy_half(&map, table, 2 * page0 + i, ring + s * stage_bytes, boxes, &full[s]);
            if (++s == a.stages) { s = 0; parity ^= 1; }
        }
        return;
    }
    int issued = 0;   // halves asked for by warp 0 (without a producer warp)
    auto issue_until = [&](int end) {
        for (; issued < min(end, 2 * (page1 - page0)); ++issued)
            latent_copy_half(&map, table, 2 * page0 + issued, ring + issued % a.stages * stage_bytes, boxes, &full[issued % a.stages]);
    };
    if (!Shape::kProducer && warp == 0) issue_until(a.stages);

    // queries as A fragments: quarter `quarter` of the width
    // quarter: 16 of the 64 values of every box, so that a warp's fragments lie at constant distances
    const int quarter = warp & 3, group = warp >> 2;
    uint32_t q[KS][MT][4];
    {
        const float* source[2 * MT];
#pragma unroll
        for (int i = 0; i < 2 * MT; ++i) {
            const int m = (i >> 1) * 16 + (i & 1) * 8 + (lane >> 2);
            const int64_t row = first + offset + m / a.head_chunk;
            source[i] = visible[m] > 0 ? a.query + (row * p.heads + chunk * M + m % a.head_chunk) * p.width : nullptr;
        }
#pragma unroll
        for (int i = 0; i < KS; ++i) {
            const int k = i * 64 + quarter * 16 + (lane & 3) * 2;
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int part = 0; part < 4; ++part) {
                    const float* from = source[mt * 2 + (part & 1)];
                    const int at = k + (part >> 1) * 8;
                    float2 v = make_float2(0.0f, 0.0f);
                    if (from && at < p.width) v = *reinterpret_cast<const float2*>(from + at);
                    q[i][mt][part] = pack_bf16(v.x, v.y);
                }
        }
    }
    float o[MT][VT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int v = 0; v < VT; ++v)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[mt][v][i] = 0.0f;
    constexpr int kOwn = M / kWarps;   // rows whose softmax this warp keeps; l_own is each lane's share of the sum
    float m_own[kOwn], l_own[kOwn];
#pragma unroll
    for (int r = 0; r < kOwn; ++r) { m_own[r] = -INFINITY; l_own[r] = 0.0f; }
    const float scale2 = p.scale * kLog2e;
    // Offsets inside a stage (rows of a fragment differ by multiples of 8, so the swizzle is the lane's own)
    const uint32_t key_offset = stage_offset((group * kKeyTiles * 8) % kHalf + (lane >> 4) * 8 + (lane & 7), quarter * 2 + ((lane >> 3) & 1));
    uint32_t value_offset[VT / 2];   // tiles past the latent's columns are never stored; their reads stay inside the row
#pragma unroll
    for (int v = 0; v < VT / 2; ++v) value_offset[v] = stage_offset(lane & 15, min(warp * VT + 2 * v, boxes * 8 - 2) + (lane >> 4));
    const uint32_t weight_at = smem_u32(weights + (lane & 15) * kWeightPitch + (lane >> 4) * 8);
    float* const score_at = scores + (quarter * M + (lane >> 2)) * kScorePitch + group * kKeyTiles * 8 + (lane & 3) * 2;
    constexpr int kSpan = VT >= 4 ? 4 : 2;   // value tiles worked at a time
    bool alive = true;

    int stage = 0;
    uint32_t phase = 0;
    auto step_stage = [&] { if (++stage == a.stages) { stage = 0; phase ^= 1; } };
    for (int t = page0; t < page1; ++t) {
        const int s0 = stage;
        const uint32_t phase0 = phase;
        step_stage();
        const int s1 = stage;
        const uint32_t phase1 = phase;
        step_stage();
        if (!mbar_wait(&full[s0], phase0) || !mbar_wait(&full[s1], phase1)) {
            if (lane == 0) atomicExch(a.status, B200_DEVICE_TIMEOUT);
            *static_cast<volatile int*>(gave_up) = 1;
        }
        const uint32_t half_at[2] = {smem_u32(ring + s0 * stage_bytes), smem_u32(ring + s1 * stage_bytes)};
        const uint32_t keys_at = group * kKeyTiles * 8 < kHalf ? half_at[0] : half_at[1];   // a warp's keys lie in one half
        float sc[MT][kKeyTiles][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int n = 0; n < kKeyTiles; ++n)
#pragma unroll
                for (int j = 0; j < 4; ++j) sc[mt][n][j] = 0.0f;
#pragma unroll
        for (int k = 0; k < KS; ++k) {
            if (k < boxes) {
#pragma unroll
                for (int n = 0; n < kKeyTiles; n += 2) {
                    uint32_t b[4];
                    ldsm_x4(b, keys_at + key_offset + static_cast<uint32_t>(k * kBoxBytes + n * 8 * 128));
#pragma unroll
                    for (int mt = 0; mt < MT; ++mt) {
                        mma_16816(sc[mt][n], q[k][mt], b[0], b[1]);
                        mma_16816(sc[mt][n + 1], q[k][mt], b[2], b[3]);
                    }
                }
            }
        }
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int n = 0; n < kKeyTiles; ++n) {
                float* at = score_at + mt * 16 * kScorePitch + n * 8;
                *reinterpret_cast<float2*>(at) = make_float2(sc[mt][n][0], sc[mt][n][1]);
                *reinterpret_cast<float2*>(at + 8 * kScorePitch) = make_float2(sc[mt][n][2], sc[mt][n][3]);
            }
        consumers_sync<Shape::kConsumers>();
        if (*static_cast<volatile int*>(gave_up)) { alive = false; break; }   // a page never arrived: every consumer leaves here
        if (!Shape::kProducer && warp == 0) issue_until(2 * (t - page0) + a.stages);   // every warp is past the products of the page before: its stages are free
#pragma unroll
        for (int r = 0; r < kOwn; ++r) {
            const int m = warp * kOwn + r, sees = visible[m] - t * kPage;
            float v0 = 0.0f, v1 = 0.0f;
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                const float2 part = *reinterpret_cast<const float2*>(scores + (w * M + m) * kScorePitch + lane * 2);
                v0 += part.x;
                v1 += part.y;
            }
            v0 = lane * 2 < sees ? v0 * scale2 : -INFINITY;
            v1 = lane * 2 + 1 < sees ? v1 * scale2 : -INFINITY;
            const float top = fmaxf(m_own[r], warp_max(fmaxf(v0, v1)));
            const float base = top == -INFINITY ? 0.0f : top;
            const float p0 = exp2_fast(v0 - base), p1 = exp2_fast(v1 - base), factor = exp2_fast(m_own[r] - base);
            l_own[r] = l_own[r] * factor + (p0 + p1);
            m_own[r] = top;
            if (lane == 0) shrink[m] = factor;
            uint32_t hi, lo;
            pack_planes(p0, p1, hi, lo);
            *reinterpret_cast<uint32_t*>(weights + m * kWeightPitch + lane * 2) = hi;
            *reinterpret_cast<uint32_t*>(weights + (M + m) * kWeightPitch + lane * 2) = lo;
        }
        consumers_sync<Shape::kConsumers>();
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            const float f0 = shrink[mt * 16 + (lane >> 2)], f1 = shrink[mt * 16 + (lane >> 2) + 8];
#pragma unroll
            for (int v = 0; v < VT; ++v) { o[mt][v][0] *= f0; o[mt][v][1] *= f0; o[mt][v][2] *= f1; o[mt][v][3] *= f1; }
        }
#pragma unroll
        for (int k = 0; k < kPage / 16; ++k) {
            if constexpr (Shape::kProducer) {
                if (k == 2) {   // the first half has been read to its end
                    __syncwarp();
                    if (lane == 0) mbar_arrive(&empty[s0]);
                }
            }
            uint32_t w[MT][2][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int plane = 0; plane < 2; ++plane)
                    ldsm_x4(w[mt][plane], weight_at + static_cast<uint32_t>(((plane * M + mt * 16) * kWeightPitch + k * 16) * 2));
#pragma unroll
            for (int v = 0; v < VT; v += kSpan) {
                uint32_t b[kSpan / 2][4];
#pragma unroll
                for (int i = 0; i < kSpan / 2; ++i)
                    ldsm_x4_trans(b[i], half_at[k >> 1] + value_offset[v / 2 + i] + (k & 1) * 16 * 128);
                // all tiles of one plane before the other: products that follow each other do not depend on each other
#pragma unroll
                for (int plane = 0; plane < 2; ++plane)
#pragma unroll
                    for (int i = 0; i < kSpan / 2; ++i)
#pragma unroll
                        for (int mt = 0; mt < MT; ++mt) {
                            mma_16816(o[mt][v + 2 * i], w[mt][plane], b[i][0], b[i][1]);
                            mma_16816(o[mt][v + 2 * i + 1], w[mt][plane], b[i][2], b[i][3]);
                        }
            }
        }
        if constexpr (Shape::kProducer) {
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[s1]);
        }
    }
    if (!alive) return;
#pragma unroll
    for (int r = 0; r < kOwn; ++r) l_own[r] = warp_sum(l_own[r]);
    if (lane == 0) {
#pragma unroll
        for (int r = 0; r < kOwn; ++r) { row_m[warp * kOwn + r] = m_own[r]; row_l[warp * kOwn + r] = l_own[r]; }
    }
    consumers_sync<Shape::kConsumers>();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int side = 0; side < 2; ++side) {
            const int m = mt * 16 + side * 8 + (lane >> 2);
            if (visible[m] == 0) continue;
            const int64_t row_head = static_cast<int64_t>(first + offset + m / a.head_chunk) * p.heads + chunk * M + m % a.head_chunk;
            const bool whole = a.splits == 1;
            const float factor = whole ? 1.0f / row_l[m] : 1.0f;
            float* target = whole ? a.out + row_head * p.rank : a.partial + (row_head * a.splits + split) * p.rank;
#pragma unroll
            for (int v = 0; v < VT; ++v) {
                const int column = (warp * VT + v) * 8 + (lane & 3) * 2;
                if (column < p.rank)
                    *reinterpret_cast<float2*>(target + column) = make_float2(o[mt][v][side * 2] * factor, o[mt][v][side * 2 + 1] * factor);
            }
            if (!whole && warp == 0 && (lane & 3) == 0) {
                a.partial_ml[(row_head * a.splits + split) * 2] = row_m[m];
                a.partial_ml[(row_head * a.splits + split) * 2 + 1] = row_l[m];
            }
        }
}

// out[row_head, :] from the splits' (max, sum, unscaled accumulator); one CTA per (row, head)
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* partial, const float* ml, int splits, int rank, float* out) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t at = blockIdx.x;
    float top = -INFINITY;
    for (int s = 0; s < splits; ++s) top = fmaxf(top, ml[(at * splits + s) * 2]);
    float total = 0.0f;
    for (int s = 0; s < splits; ++s) total += ml[(at * splits + s) * 2 + 1] * exp2f(ml[(at * splits + s) * 2] - top);
    const float inverse = 1.0f / total;
    for (int c = threadIdx.x; c < rank; c += blockDim.x) {
        float v = 0.0f;
        for (int s = 0; s < splits; ++s) {
            const float factor = exp2f(ml[(at * splits + s) * 2] - top);
            if (factor > 0.0f) v = fmaf(partial[(at * splits + s) * rank + c], factor, v);
        }
        out[at * rank + c] = v * inverse;
    }
}

constexpr int kGenericThreads = 128, kGenericKeys = 128;
// grid (heads, rows): f32 FMAs over the cached values of either dtype
__global__ void __launch_bounds__(kGenericThreads) latent_generic_kernel(const __grid_constant__ LatentAttention a) {
    extern __shared__ __align__(16) float sm[];   // query [width], accumulator [rank], weights [keys], scratch
    const LatentParams& p = a.latent;
    float* query = sm;
    float* acc = query + p.width;
    float* w = acc + p.rank;
    float* scratch = w + kGenericKeys;
    int64_t* where = reinterpret_cast<int64_t*>(scratch + 32 + ((p.width + p.rank) & 1));   // [keys] 8-byte aligned
    grid_dependency_wait();
    grid_launch_dependents();
    const int head = blockIdx.x, row = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const RowPlace place = row_place(a.rows, row);
    const int64_t row_head = static_cast<int64_t>(row) * p.heads + head;
    for (int c = threadIdx.x; c < p.width; c += kGenericThreads) query[c] = a.query[row_head * p.width + c];
    for (int c = threadIdx.x; c < p.rank; c += kGenericThreads) acc[c] = 0.0f;
    float top = -INFINITY, total = 0.0f;
    const int keys = place.position + 1;
    for (int k0 = 0; k0 < keys; k0 += kGenericKeys) {
        const int n = min(kGenericKeys, keys - k0);
        __syncthreads();
        if (threadIdx.x < n) where[threadIdx.x] = kv_offset(p.kv, place.slot, k0 + threadIdx.x, 0);
        __syncthreads();
        for (int j = warp; j < n; j += kGenericThreads / 32) {
            float dot = 0.0f;
            for (int c = lane; c < p.width; c += 32) dot = fmaf(query[c], kv_load(p.kv, 0, where[j] + c), dot);
            dot = warp_sum(dot);
            if (lane == 0) w[j] = dot * p.scale;
        }
        __syncthreads();
        float local = -INFINITY;
        for (int j = 0; j < n; ++j) local = fmaxf(local, w[j]);
        const float next = fmaxf(top, local), factor = expf(top - next);
        __syncthreads();
        if (threadIdx.x < n) w[threadIdx.x] = expf(w[threadIdx.x] - next);
        const float sum = block_sum(threadIdx.x < n ? w[threadIdx.x] : 0.0f, scratch);
        total = total * factor + sum;
        top = next;
        for (int c = threadIdx.x; c < p.rank; c += kGenericThreads) {
            float v = acc[c] * factor;
            for (int j = 0; j < n; ++j) v = fmaf(w[j], kv_load(p.kv, 0, where[j] + c), v);
            acc[c] = v;
        }
    }
    const float inverse = 1.0f / total;
    for (int c = threadIdx.x; c < p.rank; c += kGenericThreads) a.out[row_head * p.rank + c] = acc[c] * inverse;
}

bool latent_takes_mma(const LatentParams& p) {
    return p.kv.dtype == B200_BF16 && p.kv.page_size == kPage && p.kv.head_dim % 8 == 0 && p.rank % 8 == 0 && p.rank <= 512 && p.width <= 576;
}
// Rows of an item: 16 for decode steps of up to 16 heads, 32 otherwise.
int latent_tile(const LatentParams& p, int max_count) { return max_count == 1 && p.heads <= 16 ? 16 : 32; }

int latent_splits(const LatentParams& p, int sequences, int max_count, int max_length) {
    if (max_count > 1) return 1;
    int device = 0;
    if (cudaGetDevice(&device) != cudaSuccess) { cudaGetLastError(); device = -1; }
    const int sms = sm_count(device), tile = latent_tile(p, max_count);
    const int64_t items = static_cast<int64_t>(sequences) * ((p.heads + tile - 1) / tile);
    const int pages = std::max(1, (max_length + kPage - 1) / kPage);
    // rounds of CTAs x (pages of one + its fixed cost in pages), plus the merge
    int best = 1;
    double best_cost = 1e30;
    for (int s = 1; s <= std::min(64, pages); ++s) {
        const double rounds = static_cast<double>((items * s + sms - 1) / sms);
        const double cost = rounds * ((pages + s - 1) / s + 1.5) + (s > 1 ? 2.0 + 0.05 * s : 0.0);
        if (cost < best_cost - 1e-9) { best_cost = cost; best = s; }
    }
    return best;
}

template <int KS, int VT, int MT> int launch_latent_mma(LatentAttention& a, const CUtensorMap& map, int sequences, int max_count, cudaStream_t stream) {
    constexpr int M = 16 * MT;
    const LatentParams& p = a.latent;
    const int stage = (p.width + 63) / 64 * kBoxBytes, fixed = latent_fixed_bytes(M) + 1024;
    a.stages = std::min(8, (227 * 1024 - fixed) / stage);
    if (a.stages < 4) { set_error("latent attention: two pages of width %d do not fit shared memory", p.width); return B200_UNSUPPORTED; }
    const int smem = fixed + a.stages * stage;
    a.head_chunk = std::min(p.heads, M);
    a.head_chunks = (p.heads + M - 1) / M;
    a.positions_per_item = max_count == 1 ? 1 : std::max(1, M / a.head_chunk);
    auto kernel = latent_mma_kernel<KS, VT, MT>;
    B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    const dim3 grid(static_cast<unsigned>((max_count + a.positions_per_item - 1) / a.positions_per_item), static_cast<unsigned>(sequences),
                    static_cast<unsigned>(a.head_chunks * a.splits));
    return cuda_status(launch_dependent(kernel, grid, dim3(LatentShape<MT>::kThreads), smem, stream, a, map), "latent_mma_kernel launch");
}
template <int MT> int pick_latent_mma(LatentAttention& a, const CUtensorMap& map, int sequences, int max_count, cudaStream_t stream) {
    const LatentParams& p = a.latent;
    constexpr int kPer = 8 * LatentShape<MT>::kWarps;   // latent columns of one tile per warp
    if (p.rank <= 128 && p.width <= 192) return launch_latent_mma<3, 2, MT>(a, map, sequences, max_count, stream);
    if (p.rank <= 256 && p.width <= 320) return launch_latent_mma<5, 256 / kPer, MT>(a, map, sequences, max_count, stream);
    return launch_latent_mma<9, 512 / kPer, MT>(a, map, sequences, max_count, stream);
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_latent_prepare(const b200_latent_args* args, const b200_rows* pass, const float* projected, float* q_latent, void* q_hi, void* q_lo,
                        void* stream) {
    LatentParams p;
    RowsView rows;
    if (!latent_params(args, p, true) || !rows_view(pass, rows)) return B200_BAD_ARGUMENT;
    if (!projected || (!q_latent && !q_hi)) { set_error("b200_latent_prepare: operands missing"); return B200_BAD_ARGUMENT; }
    const int64_t stride = static_cast<int64_t>(p.q_rank) + p.width + static_cast<int64_t>(p.heads) * p.vdim;
    return cuda_status(launch_dependent(latent_prepare_kernel, dim3(static_cast<unsigned>(rows.rows)), dim3(256), 0, as_stream(stream), p, rows,
                                        projected, stride, q_latent, static_cast<__nv_bfloat16*>(q_hi), static_cast<__nv_bfloat16*>(q_lo)),
                       "latent_prepare_kernel launch");
}

int b200_latent_query(const b200_latent_args* args, const b200_rows* pass, const float* query, float* absorbed, void* stream) {
    HeadLinear h{};
    if (!latent_params(args, h.latent, false) || !rows_view(pass, h.rows)) return B200_BAD_ARGUMENT;
    if (!query || !absorbed) { set_error("b200_latent_query: operands missing"); return B200_BAD_ARGUMENT; }
    const LatentParams& p = h.latent;
    h.x = query; h.x_head = p.dim + p.rot_dim; h.x_row = h.x_head * p.heads;
    h.row_count = h.rows.rows; h.in = p.dim; h.out = p.rank; h.w = p.w_key; h.query = true; h.y = absorbed;
    return launch_head_linear(h, as_stream(stream));
}

int b200_latent_value(const b200_latent_args* args, int64_t rows, const float* latent, const float* gate, int64_t gate_stride, float* out,
                      void* out_hi, void* out_lo, void* stream) {
    HeadLinear h{};
    if (!latent_params(args, h.latent, false)) return B200_BAD_ARGUMENT;
    if (!latent || !gate || rows < 0 || rows > INT32_MAX || (!out && !out_hi)) { set_error("b200_latent_value: operands missing"); return B200_BAD_ARGUMENT; }
    if (rows == 0) return B200_OK;
    const LatentParams& p = h.latent;
    h.x = latent; h.x_head = p.rank; h.x_row = static_cast<int64_t>(p.rank) * p.heads;
    h.row_count = static_cast<int>(rows); h.in = p.rank; h.out = p.vdim; h.w = p.w_value;
    h.y = out; h.gate = gate; h.gate_stride = gate_stride;
    h.out_hi = static_cast<__nv_bfloat16*>(out_hi); h.out_lo = static_cast<__nv_bfloat16*>(out_lo);
    return launch_head_linear(h, as_stream(stream));
}

size_t b200_latent_scratch_bytes(const b200_latent_args* args, int64_t rows, int32_t sequences, int32_t max_count, int32_t max_length) {
    LatentParams p;
    if (!latent_params(args, p, true) || rows <= 0 || !latent_takes_mma(p)) return 0;
    const int splits = latent_splits(p, sequences, max_count, max_length);
    return splits > 1 ? static_cast<size_t>(rows) * p.heads * splits * (p.rank + 2) * sizeof(float) : 0;
}

const char* b200_latent_attention_kernel(const b200_latent_args* args) {
    LatentParams p;
    return latent_params(args, p, true) ? (latent_takes_mma(p) ? "latent_mma_kernel" : "latent_generic_kernel") : "";
}

int b200_latent_attention(const b200_latent_args* args, const b200_rows* pass, const float* absorbed, int32_t max_length, void* scratch,
                          size_t scratch_bytes, float* latent_out, void* stream) {
    LatentAttention a{};
    if (!latent_params(args, a.latent, true) || !rows_view(pass, a.rows)) return B200_BAD_ARGUMENT;
    if (!absorbed || !latent_out || max_length <= 0) { set_error("b200_latent_attention: operands missing"); return B200_BAD_ARGUMENT; }
    const LatentParams& p = a.latent;
    a.query = absorbed; a.out = latent_out;
    if (!latent_takes_mma(p)) {
        const size_t smem = sizeof(float) * (p.width + p.rank + kGenericKeys + 32 + 2) + sizeof(int64_t) * kGenericKeys;
        if (smem > 200 * 1024 || a.rows.rows > 65535) { set_error("latent attention: sizes outside the generic kernel"); return B200_UNSUPPORTED; }
        if (smem > 46 * 1024) B200_CUDA(cudaFuncSetAttribute(latent_generic_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        return cuda_status(launch_dependent(latent_generic_kernel, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(a.rows.rows)),
                                            dim3(kGenericThreads), smem, as_stream(stream), a), "latent_generic_kernel launch");
    }
    int device = 0;
    B200_CUDA(cudaGetDevice(&device));
    a.status = device_status_word(device);
    if (!a.status) { set_error("the device status word could not be allocated"); return B200_NO_DEVICE; }
    a.splits = latent_splits(p, a.rows.sequences, a.rows.max_count, max_length);
    if (a.rows.sequences > 65535) { set_error("latent attention: too many sequences in one pass"); return B200_UNSUPPORTED; }
    if (a.splits > 1) {
        const size_t pairs = static_cast<size_t>(a.rows.rows) * p.heads * a.splits;
        if (!scratch || scratch_bytes < pairs * (p.rank + 2) * sizeof(float)) { set_error("latent attention: scratch too small"); return B200_BAD_ARGUMENT; }
        a.partial = static_cast<float*>(scratch);
        a.partial_ml = a.partial + pairs * p.rank;
    }
    const int sequences = a.rows.sequences, max_count = a.rows.max_count;
    const CUtensorMap* map = kv_tensor_map(args->cache, 0);
    if (!map) { set_error("latent attention: the cache has no tensor map"); return B200_UNSUPPORTED; }
    const int status = latent_tile(p, max_count) == 16 ? pick_latent_mma<1>(a, *map, sequences, max_count, as_stream(stream))
                                                       : pick_latent_mma<2>(a, *map, sequences, max_count, as_stream(stream));
    if (status != B200_OK || a.splits == 1) return status;
    return cuda_status(launch_dependent(latent_combine_kernel, dim3(static_cast<unsigned>(a.rows.rows * p.heads)), dim3(128), 0, as_stream(stream),
                                        static_cast<const float*>(a.partial), static_cast<const float*>(a.partial_ml), a.splits, p.rank, a.out),
                       "latent_combine_kernel launch");
}

}  // extern "C"
