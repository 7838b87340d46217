// Gated delta rule.  Per head, with key and query of unit length (the query also over sqrt(state)):
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// Everything is f32.  The convolved channels [v | k | q], the decay's column and the state's place are those of a state-space layer
// (state_space.cuh: x, B, C; S[state][vdim]); beta's columns follow the decays'.  Both products with the state are taken of the state as
// it was, so that one sweep and one reduction serve a token:
//     o = g S_old^T q + (k . q) u
// and the lengths of k and q enter as factors of the sums, so the channels are never normed in memory.
//
//   * delta_step_kernel, one CTA per (sequence, head): convolution inside, the state in registers between the two sweeps.
//   * delta_step_stream_kernel (large batches; the convolution as its own kernel): persistent CTAs, states by bulk copies through two
//     stages, as in ssm_step_stream_kernel.
//   * delta_scan_kernel (longer passes): the state in registers across the pass, eight (or 32) lanes along the state dimension, four value
//     columns per lane; the sums of a token's two products are exchanged so that every lane ends with one of them.
#include "state_space.cuh"

#include <algorithm>

namespace b200 {
namespace {

constexpr float kUnitEps = 1e-6f;

// Factors of a token: decay, step size, lengths' reciprocals of key and query (the latter over sqrt(state)), and k . q of the unit vectors.
struct DeltaFactors { float decay, beta, key, query, both; };
__device__ __forceinline__ DeltaFactors delta_factors(const SsmParams& p, float decay, float beta, float kk, float qq, float kq) {
    const float key = 1.0f / sqrtf(kk + kUnitEps), query = 1.0f / (sqrtf(qq + kUnitEps) * sqrtf(static_cast<float>(p.state)));
    return {decay, beta, key, query, kq * key * query};
}
__device__ __forceinline__ float beta_of(const SsmParams& p, const float* row, int head) {
    return sigmoid_exact(row[p.heads * p.vdim + p.channels + p.heads + head]);
}
// |k|^2, |q|^2 and k . q of a token, by one warp; every lane gets them.
__device__ __forceinline__ float3 key_query_sums(const float* k, const float* q, int n, int lane) {
    float3 s = make_float3(0.0f, 0.0f, 0.0f);
    for (int i = lane; i < n; i += 32) {
        const float a = k[i], b = q[i];
        s.x = fmaf(a, a, s.x);
        s.y = fmaf(b, b, s.y);
        s.z = fmaf(a, b, s.z);
    }
    return make_float3(warp_sum(s.x), warp_sum(s.y), warp_sum(s.z));
}

constexpr int kDeltaKeep = 16;   // state rows that a thread of the step kernel keeps between its sweeps; the rest is read twice

// grid (heads, sequences); one row per sequence.  V = 4 when vdim is a multiple of 4.
template <int V>
__global__ void __launch_bounds__(kStepThreads, 2) delta_step_kernel(const SsmParams p, const RowsView rows) {
    extern __shared__ __align__(16) float sm[];   // [v: vdim | k: state | q: state], partial sums 2 x [threads * V], written values [vdim]
    const int P = p.vdim, N = p.state, head = blockIdx.x, row = blockIdx.y, inner = p.heads * P;
    float* mixed = sm;
    float* partial = sm + ((P + 2 * N + 3) & ~3);
    float* written = partial + 2 * kStepThreads * V;
    grid_dependency_wait();
    grid_launch_dependents();
    const int slot = __ldg(rows.slot + row), position = rows.lengths[slot];
    const float* in = p.projected + static_cast<int64_t>(row) * p.stride;
    const bool fresh = position == 0;
    float* state = p.ssm_state + (static_cast<int64_t>(slot) * p.heads + head) * N * P;

    const int columns = P / V, slices = kStepThreads / columns > 0 ? kStepThreads / columns : 1;
    const int slice = columns <= kStepThreads ? static_cast<int>(threadIdx.x) / columns : 0, own = static_cast<int>(threadIdx.x) - slice * columns;
    Lanes<V> s[kDeltaKeep];
    auto fetch_row = [&](int n, int column) {
        Lanes<V> r;
#pragma unroll
        for (int k = 0; k < V; ++k) r.v[k] = 0.0f;
        if (!fresh && n < N) r = load_lanes<V>(state + static_cast<int64_t>(n) * P + column * V);
        return r;
    };
    auto fetch = [&](int column, bool active) {
#pragma unroll
        for (int i = 0; i < kDeltaKeep; ++i) s[i] = fetch_row(active ? slice + i * slices : N, column);
    };
    fetch(own, own < columns && slice < slices);

    convolve_head(p, in, slot, position, head, mixed);
    const float decay = step_rate(p, in, head).decay, beta = beta_of(p, in, head);
    __syncthreads();
    const float *value = mixed, *key = mixed + P, *query = mixed + P + N;
    const float3 sums = key_query_sums(key, query, N, threadIdx.x & 31);
    const DeltaFactors f = delta_factors(p, decay, beta, sums.x, sums.y, sums.z);

    for (int base = 0; base < columns; base += kStepThreads) {
        const int column = base + own;
        const bool active = column < columns && slice < slices;
        if (base > 0) fetch(column, active);
        Lanes<V> by_key, by_query;
#pragma unroll
        for (int k = 0; k < V; ++k) by_key.v[k] = by_query.v[k] = 0.0f;
        auto add = [&](const Lanes<V>& v, int n) {
            const float a = key[n], b = query[n];
#pragma unroll
            for (int k = 0; k < V; ++k) {
                by_key.v[k] = fmaf(v.v[k], a, by_key.v[k]);
                by_query.v[k] = fmaf(v.v[k], b, by_query.v[k]);
            }
        };
        if (active) {
#pragma unroll
            for (int i = 0; i < kDeltaKeep; ++i)
                if (slice + i * slices < N) add(s[i], slice + i * slices);
            for (int n = slice + kDeltaKeep * slices; n < N; n += slices) add(fetch_row(n, column), n);
        }
        __syncthreads();
        store_lanes<V>(partial + threadIdx.x * V, by_key);
        store_lanes<V>(partial + (kStepThreads + threadIdx.x) * V, by_query);
        __syncthreads();
        const int width = columns <= kStepThreads ? columns : min(kStepThreads, columns - base), stride = columns <= kStepThreads ? columns * V : 0;
        for (int i = threadIdx.x; i < width * V; i += kStepThreads) {
            float of_key = 0.0f, of_query = 0.0f;
            for (int k = 0; k < slices; ++k) {
                of_key += partial[k * stride + i];
                of_query += partial[kStepThreads * V + k * stride + i];
            }
            const int at = base * V + i;
            const float u = f.beta * (value[at] - f.decay * f.key * of_key);
            written[i] = u * f.key;
            p.y[static_cast<int64_t>(row) * inner + head * P + at] = fmaf(f.both, u, f.decay * f.query * of_query);
        }
        __syncthreads();
        if (active) {
            const Lanes<V> w = load_lanes<V>(written + own * V);
            auto update = [&](Lanes<V> v, int n) {
                const float a = key[n];
#pragma unroll
                for (int k = 0; k < V; ++k) v.v[k] = fmaf(v.v[k], f.decay, a * w.v[k]);
                store_lanes<V>(state + static_cast<int64_t>(n) * P + column * V, v);
            };
#pragma unroll
            for (int i = 0; i < kDeltaKeep; ++i)
                if (slice + i * slices < N) update(s[i], slice + i * slices);
            for (int n = slice + kDeltaKeep * slices; n < N; n += slices) update(fetch_row(n, column), n);
        }
    }
}

// ---- streamed step --------------------------------------------------------------------------------------------------
constexpr int kStreamThreads = kStepThreads + 32;
struct DeltaMeta { float decay, beta, fresh; };
size_t delta_stream_bytes(int state, int vdim) {
    return sizeof(float) * (2 * (static_cast<size_t>(state) * vdim + vdim + 2 * state) + 2 * kStepThreads * 4 + vdim);
}

// Persistent CTAs walk the (sequence, head) pairs; vdim and state multiples of 4, vdim at most 1024.
__global__ void __launch_bounds__(kStreamThreads) delta_step_stream_kernel(const SsmParams p, const RowsView rows, int32_t* status) {
    extern __shared__ __align__(16) float sm[];   // 2 x [state * vdim | v | k | q], partial sums 2 x [threads * 4], written values [vdim]
    __shared__ uint64_t full[2], done[2];
    __shared__ DeltaMeta meta[2];
    __shared__ int gave_up;
    const int P = p.vdim, N = p.state, inner = p.heads * P, block = N * P, stage_floats = block + P + 2 * N, columns = P >> 2,
              slices = kStepThreads / columns;
    const int units = rows.rows * p.heads;
    float* partial = sm + 2 * stage_floats;
    float* written = partial + 2 * kStepThreads * 4;
    if (threadIdx.x == 0) {
        for (int s = 0; s < 2; ++s) { mbar_init(&full[s], 1); mbar_init(&done[s], kStepThreads); }
        mbar_fence_init();
        gave_up = 0;
    }
    grid_dependency_wait();
    grid_launch_dependents();
    __syncthreads();

    if (threadIdx.x >= kStepThreads) {   // producer warp; one lane issues
        if ((threadIdx.x & 31) != 0) return;
        float* pending[2] = {nullptr, nullptr};
        int turn = 0;
        for (int unit = blockIdx.x; unit < units + 2 * static_cast<int>(gridDim.x); unit += gridDim.x, ++turn) {
            const int stage = turn & 1, row = unit / p.heads, head = unit - row * p.heads;
            const bool live = unit < units;
            float* state = nullptr;
            float decay = 0.0f, beta = 0.0f;
            bool fresh = true;
            if (live) {   // operands of this pair, while the stage may still be in use
                const int slot = __ldg(rows.slot + row);
                fresh = rows.lengths[slot] == 0;
                state = p.ssm_state + (static_cast<int64_t>(slot) * p.heads + head) * block;
                const float* in = p.projected + static_cast<int64_t>(row) * p.stride;
                decay = step_rate(p, in, head).decay;
                beta = beta_of(p, in, head);
            }
            if (turn >= 2 && pending[stage]) {   // the pair two turns ago has been worked on: its state goes back
                if (!mbar_wait(&done[stage], ((turn >> 1) - 1) & 1)) {
                    atomicExch(status, B200_DEVICE_TIMEOUT);
                    break;
                }
                bulk_store(pending[stage], sm + stage * stage_floats, static_cast<uint32_t>(block) * 4);
                asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
            }
            pending[stage] = state;
            if (!live) continue;
            float* at = sm + stage * stage_floats;
            meta[stage] = DeltaMeta{decay, beta, fresh ? 1.0f : 0.0f};
            mbar_expect_tx(&full[stage], static_cast<uint32_t>((fresh ? 0 : block) + P + 2 * N) * 4);
            if (!fresh) bulk_load(at, state, static_cast<uint32_t>(block) * 4, &full[stage]);
            const float* mixed = p.mixed + static_cast<int64_t>(row) * p.channels;
            const int group = head / (p.heads / p.groups);
            bulk_load(at + block, mixed + head * P, static_cast<uint32_t>(P) * 4, &full[stage]);
            bulk_load(at + block + P, mixed + inner + group * N, static_cast<uint32_t>(N) * 4, &full[stage]);
            bulk_load(at + block + P + N, mixed + inner + (p.groups + group) * N, static_cast<uint32_t>(N) * 4, &full[stage]);
        }
        asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
        return;
    }

    const int slice = static_cast<int>(threadIdx.x) / columns, column = static_cast<int>(threadIdx.x) - slice * columns;
    const bool active = slice < slices;
    int turn = 0;
    for (int unit = blockIdx.x; unit < units; unit += gridDim.x, ++turn) {
        const int stage = turn & 1, row = unit / p.heads, head = unit - row * p.heads;
        const bool arrived = mbar_wait(&full[stage], (turn >> 1) & 1);
        if (!arrived) {
            if ((threadIdx.x & 31) == 0) atomicExch(status, B200_DEVICE_TIMEOUT);
            *static_cast<volatile int*>(&gave_up) = 1;
        }
        const DeltaMeta m = meta[stage];
        float* at = sm + stage * stage_floats;
        const float *value = at + block, *key = value + P, *query = key + N;
        const bool fresh = m.fresh != 0.0f;
        const float3 sums = key_query_sums(key, query, N, threadIdx.x & 31);
        const DeltaFactors f = delta_factors(p, m.decay, m.beta, sums.x, sums.y, sums.z);
        float4* s = reinterpret_cast<float4*>(at) + column;
        float4 by_key = make_float4(0.0f, 0.0f, 0.0f, 0.0f), by_query = by_key;
        if (active && arrived && !fresh) {
#pragma unroll 8
            for (int n = slice; n < N; n += slices) {
                const float a = key[n], b = query[n];
                const float4 v = s[n * columns];
                by_key = make_float4(fmaf(v.x, a, by_key.x), fmaf(v.y, a, by_key.y), fmaf(v.z, a, by_key.z), fmaf(v.w, a, by_key.w));
                by_query = make_float4(fmaf(v.x, b, by_query.x), fmaf(v.y, b, by_query.y), fmaf(v.z, b, by_query.z), fmaf(v.w, b, by_query.w));
            }
        }
        reinterpret_cast<float4*>(partial)[threadIdx.x] = by_key;
        reinterpret_cast<float4*>(partial)[kStepThreads + threadIdx.x] = by_query;
        asm volatile("bar.sync 1, %0;" ::"n"(kStepThreads) : "memory");
        if (*static_cast<volatile int*>(&gave_up)) return;   // a state never arrived: the eight warps leave together
        for (int i = threadIdx.x; i < P; i += kStepThreads) {
            float of_key = 0.0f, of_query = 0.0f;
            for (int k = 0; k < slices; ++k) {
                of_key += partial[k * P + i];
                of_query += partial[kStepThreads * 4 + k * P + i];
            }
            const float u = f.beta * (value[i] - f.decay * f.key * of_key);
            written[i] = u * f.key;
            p.y[static_cast<int64_t>(row) * inner + head * P + i] = fmaf(f.both, u, f.decay * f.query * of_query);
        }
        asm volatile("bar.sync 1, %0;" ::"n"(kStepThreads) : "memory");
        if (active) {
            const float4 w = reinterpret_cast<const float4*>(written)[column];
#pragma unroll 8
            for (int n = slice; n < N; n += slices) {
                const float a = key[n];
                float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (!fresh) v = s[n * columns];
                s[n * columns] = make_float4(fmaf(v.x, f.decay, a * w.x), fmaf(v.y, f.decay, a * w.y), fmaf(v.z, f.decay, a * w.z), fmaf(v.w, f.decay, a * w.w));
            }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // the updated state is read by the copy engine
        mbar_arrive(&done[stage]);
    }
}

// ---- scan -----------------------------------------------------------------------------------------------------------
constexpr int kDeltaWarps = 4;

// LN (8 or 32) lanes of a warp share the state dimension (4 * Q values each, in quads LN * 4 apart), the other 32 / LN lane groups hold
// four value columns each.  grid (column tiles, heads, sequences).
template <int LN, int Q>
__global__ void __launch_bounds__(kDeltaWarps * 32, LN * Q <= 32 ? 3 : 2) delta_scan_kernel(const SsmParams p, const RowsView rows) {
    static_assert(LN == 8 || LN == 32);
    constexpr int kNp = LN * 4 * Q;                       // padded state size
    constexpr int kTokens = kNp <= 128 ? 16 : 4;          // tokens staged at a time
    constexpr int kGroups = 32 / LN;
    constexpr int kColumns = kDeltaWarps * kGroups * 4;   // value columns of the CTA
    __shared__ __align__(16) float sk[2][kTokens][kNp], sq[2][kTokens][kNp], sv[2][kTokens][kColumns];
    __shared__ float srate[2][kTokens], sbeta[2][kTokens];
    __shared__ DeltaFactors factors[kTokens];
    grid_dependency_wait();
    grid_launch_dependents();
    const int P = p.vdim, N = p.state, head = blockIdx.y, sequence = blockIdx.z, column0 = blockIdx.x * kColumns;
    const int group = head / (p.heads / p.groups), inner = p.heads * P;
    const int first = __ldg(rows.first + sequence), count = __ldg(rows.first + sequence + 1) - first, slot = __ldg(rows.slot + sequence);
    const bool fresh = rows.lengths[slot] == 0;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ln = lane % LN, lg = lane / LN;
    const int local = (warp * kGroups + lg) * 4, column = column0 + local;   // first of this lane's four value columns
    float* state = p.ssm_state + (static_cast<int64_t>(slot) * p.heads + head) * N * P;

    for (int i = threadIdx.x; i < 2 * kTokens * kNp; i += blockDim.x) { (&sk[0][0][0])[i] = 0.0f; (&sq[0][0][0])[i] = 0.0f; }
    for (int i = threadIdx.x; i < 2 * kTokens * kColumns; i += blockDim.x) (&sv[0][0][0])[i] = 0.0f;
    __syncthreads();

    uint64_t S[4][2 * Q];
#pragma unroll
    for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int q = 0; q < 2 * Q; ++q) {
            const int n = (q >> 1) * LN * 4 + ln * 4 + (q & 1) * 2;
            float a = 0.0f, b = 0.0f;
            if (!fresh && column + k < P) {
                if (n < N) a = state[static_cast<int64_t>(n) * P + column + k];
                if (n + 1 < N) b = state[static_cast<int64_t>(n + 1) * P + column + k];
            }
            S[k][q] = pack2(a, b);
        }
    const float rate = -expf(p.a_log[head]), dt_bias = p.dt_bias[head];
    const int live_columns = min(kColumns, P - column0);
    const bool aligned = ((p.channels | P | N | inner) & 3) == 0 && (reinterpret_cast<uintptr_t>(p.mixed) & 15) == 0;

    auto stage = [&](int chunk) {
        const int buffer = chunk & 1, t0 = chunk * kTokens, tokens = min(kTokens, count - t0);
        const float* from[3] = {p.mixed + head * P + column0, p.mixed + inner + group * N, p.mixed + inner + (p.groups + group) * N};
        const int width[3] = {live_columns, N, N};
        for (int t = warp; t < tokens; t += kDeltaWarps) {
            const int64_t row = static_cast<int64_t>(first + t0 + t) * p.channels;
            float* to[3] = {sv[buffer][t], sk[buffer][t], sq[buffer][t]};
#pragma unroll
            for (int part = 0; part < 3; ++part) {
                if (aligned) {
                    for (int c = lane * 4; c < width[part]; c += 128) copy_async_16(smem_u32(to[part] + c), from[part] + row + c, true);
                } else {
                    for (int c = lane; c < width[part]; c += 32) copy_async_4(to[part] + c, from[part] + row + c);
                }
            }
        }
        if (threadIdx.x < tokens) {
            const float* rates = p.projected + static_cast<int64_t>(first + t0 + threadIdx.x) * p.stride + inner + p.channels + head;
            copy_async_4(&srate[buffer][threadIdx.x], rates);
            copy_async_4(&sbeta[buffer][threadIdx.x], rates + p.heads);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    const int chunks = (count + kTokens - 1) / kTokens;
    // after the exchanges below a lane holds one sum: of the key (even lanes) or the query (odd lanes), for column `mine` of its four
    const bool odd = lane & 1, second = lane & 2, third = lane & 4;
    const int mine = (second ? 2 : 0) + (third ? 1 : 0), group_lane = lane & ~(LN - 1);
    const bool writes = odd && ln < 8 && column + mine < P;
    stage(0);
    for (int chunk = 0; chunk < chunks; ++chunk) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                  // the chunk has landed; the other buffer and the factors are free
        if (chunk + 1 < chunks) stage(chunk + 1);
        const int buffer = chunk & 1, t0 = chunk * kTokens, tokens = min(kTokens, count - t0);
        for (int t = warp; t < tokens; t += kDeltaWarps) {
            const float3 sums = key_query_sums(sk[buffer][t], sq[buffer][t], N, lane);
            if (lane == 0)
                factors[t] = delta_factors(p, expf(rate * softplus(srate[buffer][t] + dt_bias)), sigmoid_exact(sbeta[buffer][t]), sums.x, sums.y, sums.z);
        }
        __syncthreads();
        float* const y_chunk = p.y + static_cast<int64_t>(first + t0) * inner + head * P + column + mine;
        auto token = [&](int t) {
            const DeltaFactors f = factors[t];
            const float v = sv[buffer][t][local + mine];
            ulonglong2 k[Q];
            uint64_t by_key[4], by_query[4];
#pragma unroll
            for (int q = 0; q < Q; ++q) {
                k[q] = *reinterpret_cast<const ulonglong2*>(&sk[buffer][t][q * LN * 4 + ln * 4]);
                const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(&sq[buffer][t][q * LN * 4 + ln * 4]);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    by_key[c] = q == 0 ? mul2(S[c][0], k[0].x) : fma2(S[c][2 * q], k[q].x, by_key[c]);
                    by_query[c] = q == 0 ? mul2(S[c][0], b.x) : fma2(S[c][2 * q], b.x, by_query[c]);
                    by_key[c] = fma2(S[c][2 * q + 1], k[q].y, by_key[c]);
                    by_query[c] = fma2(S[c][2 * q + 1], b.y, by_query[c]);
                }
            }
            // eight sums over the lanes of the group: each exchange halves what a lane still carries
            float four[4], two[2];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float2 a = unpack2(by_key[c]), b = unpack2(by_query[c]);
                const float of_key = a.x + a.y, of_query = b.x + b.y;
                four[c] = (odd ? of_query : of_key) + __shfl_xor_sync(0xffffffffu, odd ? of_key : of_query, 1);
            }
#pragma unroll
            for (int c = 0; c < 2; ++c) two[c] = (second ? four[2 + c] : four[c]) + __shfl_xor_sync(0xffffffffu, second ? four[c] : four[2 + c], 2);
            float one = (third ? two[1] : two[0]) + __shfl_xor_sync(0xffffffffu, third ? two[0] : two[1], 4);
#pragma unroll
            for (int o = 8; o < LN; o <<= 1) one += __shfl_xor_sync(0xffffffffu, one, o);
            // even lanes: the value that is written for their column; the group's lanes hand all four around
            const float u = f.beta * (v - f.decay * f.key * one);
            const uint64_t decay2 = pack2(f.decay, f.decay);
            float own = 0.0f;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float uc = __shfl_sync(0xffffffffu, u, group_lane + ((c >> 1) << 1) + ((c & 1) << 2));
                if (c == mine) own = uc;
                const float w = uc * f.key;
                const uint64_t w2 = pack2(w, w);
#pragma unroll
                for (int q = 0; q < Q; ++q) {
                    S[c][2 * q] = fma2(S[c][2 * q], decay2, mul2(w2, k[q].x));
                    S[c][2 * q + 1] = fma2(S[c][2 * q + 1], decay2, mul2(w2, k[q].y));
                }
            }
            if (writes) y_chunk[static_cast<int64_t>(t) * inner] = fmaf(f.both, own, f.decay * f.query * one);
        };
        if (tokens == kTokens) {
#pragma unroll 2
            for (int t = 0; t < kTokens; ++t) token(t);
        } else {
            for (int t = 0; t < tokens; ++t) token(t);
        }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int q = 0; q < 2 * Q; ++q) {
            const int n = (q >> 1) * LN * 4 + ln * 4 + (q & 1) * 2;
            const float2 v = unpack2(S[k][q]);
            if (column + k < P) {
                if (n < N) state[static_cast<int64_t>(n) * P + column + k] = v.x;
                if (n + 1 < N) state[static_cast<int64_t>(n + 1) * P + column + k] = v.y;
            }
        }
}

template <int LN, int Q> int launch_scan(const SsmParams& p, const RowsView& rows, cudaStream_t stream) {
    constexpr int kColumns = kDeltaWarps * (32 / LN) * 4;
    const dim3 grid(static_cast<unsigned>((p.vdim + kColumns - 1) / kColumns), static_cast<unsigned>(p.heads), static_cast<unsigned>(rows.sequences));
    return cuda_status(launch_dependent(delta_scan_kernel<LN, Q>, grid, dim3(kDeltaWarps * 32), 0, stream, p, rows), "delta_scan_kernel launch");
}

}  // namespace

int launch_delta_step(const SsmParams& p, const RowsView& rows, cudaStream_t stream) {
    const bool quads = p.vdim % 4 == 0 && (reinterpret_cast<uintptr_t>(p.ssm_state) & 15) == 0;
    const int wide = quads ? 4 : 1;
    const size_t smem = sizeof(float) * (((p.vdim + 2 * p.state + 3) & ~3) + 2 * kStepThreads * wide + std::min(p.vdim, kStepThreads * wide));
    if (smem > 200 * 1024) { set_error("delta rule: a head of %d x %d values does not fit shared memory", p.state, p.vdim); return B200_UNSUPPORTED; }
    auto kernel = quads ? delta_step_kernel<4> : delta_step_kernel<1>;
    if (smem > 46 * 1024) B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    return cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(rows.sequences)), dim3(kStepThreads), smem, stream, p, rows),
                       "delta_step_kernel launch");
}

namespace {
int64_t stream_ctas(const SsmParams& p, int sms) {
    return sms * std::min<int64_t>(7, (228 * 1024) / (delta_stream_bytes(p.state, p.vdim) + 1024 + 128));
}
}  // namespace

// Streaming pays from a few pairs per CTA on; below that its extra launch and ramp cost more.
bool delta_step_streams(const SsmParams& p, const RowsView& rows, int sms) {
    const bool aligned = ((reinterpret_cast<uintptr_t>(p.ssm_state) | reinterpret_cast<uintptr_t>(p.mixed)) & 15) == 0;
    return aligned && p.vdim % 4 == 0 && p.state % 4 == 0 && p.vdim <= 4 * kStepThreads && delta_stream_bytes(p.state, p.vdim) <= 200 * 1024
        && static_cast<int64_t>(rows.rows) * p.heads >= 4 * stream_ctas(p, sms);
}

int launch_delta_step_stream(const SsmParams& p, const RowsView& rows, int sms, int32_t* status, cudaStream_t stream) {
    const size_t smem = delta_stream_bytes(p.state, p.vdim);
    B200_CUDA(cudaFuncSetAttribute(delta_step_stream_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    const int64_t ctas = std::min<int64_t>(static_cast<int64_t>(rows.rows) * p.heads, stream_ctas(p, sms));
    return cuda_status(launch_dependent(delta_step_stream_kernel, dim3(static_cast<unsigned>(ctas)), dim3(kStreamThreads), smem, stream, p, rows, status),
                       "delta_step_stream_kernel launch");
}

int launch_delta_scan(const SsmParams& p, const RowsView& rows, cudaStream_t stream) {
    if (p.state <= 32) return launch_scan<8, 1>(p, rows, stream);
    if (p.state <= 64) return launch_scan<8, 2>(p, rows, stream);
    if (p.state <= 96) return launch_scan<8, 3>(p, rows, stream);
    if (p.state <= 128) return launch_scan<8, 4>(p, rows, stream);
    if (p.state <= 256) return launch_scan<32, 2>(p, rows, stream);
    return launch_scan<32, 4>(p, rows, stream);
}

}  // namespace b200
