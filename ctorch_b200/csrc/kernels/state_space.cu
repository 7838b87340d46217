// State-space layers (Mamba-2): short causal convolution, selective recurrence, gated group norm; and the small kernels of
// packed passes.  Everything here is f32: decays, step sizes, states and norms.  Lightning attention is the same recurrence with a fixed
// decay per head, a step size of one, no skip and no convolution (only its SiLU): keys for B, queries for C, values for x.  The gated delta
// rule shares the convolution and takes its own steps and scan (delta_rule.cu).
//
//   * Decode (one row per sequence): per (sequence, head) the channels the head needs are convolved from the slot's ring of recent
//     inputs, then its [state][vdim] matrix is read once - decay, add dt B x^T, partial sums of S^T C - and written back.  The layer
//     is bound by that traffic (8 bytes per state value and token): ssm_step_stream_kernel has persistent CTAs through which the
//     states stream by bulk copies; ssm_step_kernel, one CTA per pair, serves the sizes that do not fit it.
//   * Longer passes: short_conv_kernel over all rows, conv_ring_kernel (the last inputs into the slot's ring), and
//     ssm_scan_kernel: the state lives in registers across the whole pass, spread over a warp as state-dimension slices
//     x 4 value columns per lane; tokens are staged through a double-buffered shared-memory chunk; products go two at a
//     time through the packed f32 pipe.
// The ring has `taps` entries although a token needs only taps - 1 old inputs: the entry a step writes is never one that the
// same step reads, so the CTAs of a head group need no ordering among themselves.
#include "state_space.cuh"

#include <algorithm>
#include <cmath>

namespace b200 {

bool rows_view(const b200_rows* pass, RowsView& view) {
    if (!pass || pass->rows <= 0 || pass->rows > INT32_MAX || pass->sequences <= 0 || pass->sequences > pass->rows || pass->max_count <= 0
        || pass->max_count > pass->rows || !pass->slot || !pass->first || !pass->sequence || !pass->lengths) {
        set_error("inconsistent packed pass (b200_rows)");
        return false;
    }
    view = RowsView{static_cast<int>(pass->rows), pass->sequences, pass->max_count, pass->slot, pass->first, pass->sequence, pass->lengths};
    return true;
}

namespace {

__device__ __forceinline__ float skip_of(const SsmParams& p, int head) { return p.fixed_decay ? 0.0f : p.d[head]; }

// mixed[row, c] = silu(x | B | C): the inputs of a recurrence without convolution, grid (channel blocks, rows), V channels per thread.
template <int V> __global__ void __launch_bounds__(128) activate_channels_kernel(const SsmParams p) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const int64_t row = blockIdx.y;
    if (c >= p.channels) return;
    Lanes<V> v = load_lanes<V>(p.projected + row * p.stride + p.heads * p.vdim + c);
#pragma unroll
    for (int k = 0; k < V; ++k) v.v[k] *= sigmoid_exact(v.v[k]);
    store_lanes<V>(p.mixed + row * p.channels + c, v);
}
template <int V> int launch_activate(const SsmParams& p, int rows, cudaStream_t stream) {
    const dim3 grid(static_cast<unsigned>((p.channels / V + 127) / 128), static_cast<unsigned>(rows));
    return cuda_status(launch_dependent(activate_channels_kernel<V>, grid, dim3(128), 0, stream, p), "activate_channels_kernel launch");
}

// Streamed step, first half: mixed[row, c] = silu(conv(x | B | C)) of one row per sequence, and the row's inputs into the ring.
// grid (channel blocks, rows), V channels per thread.
template <int V> __global__ void __launch_bounds__(128) conv_step_kernel(const SsmParams p, const RowsView rows) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V, row = blockIdx.y, inner = p.heads * p.vdim;
    if (c >= p.channels) return;
    const int slot = __ldg(rows.slot + row), position = rows.lengths[slot], ring_at = position % p.taps;
    float* const ring = p.conv_state + static_cast<int64_t>(slot) * p.taps * p.channels + c;
    const Lanes<V> now = load_lanes<V>(p.projected + static_cast<int64_t>(row) * p.stride + inner + c);
    Lanes<V> acc = load_lanes<V>(p.conv_bias + c);
#pragma unroll 4
    for (int j = 0; j < p.taps - 1; ++j) {
        const int back = p.taps - 1 - j, at = ring_at < back ? ring_at - back + p.taps : ring_at - back;
        const Lanes<V> old = load_lanes<V>(ring + at * p.channels);   // (an unused entry before the sequence's start)
#pragma unroll
        for (int k = 0; k < V; ++k)
            acc.v[k] = fmaf(p.conv_weight[(c + k) * p.taps + j], position < back ? 0.0f : old.v[k], acc.v[k]);
    }
#pragma unroll
    for (int k = 0; k < V; ++k) {
        acc.v[k] = fmaf(p.conv_weight[(c + k) * p.taps + p.taps - 1], now.v[k], acc.v[k]);
        acc.v[k] *= sigmoid_exact(acc.v[k]);
    }
    store_lanes<V>(ring + ring_at * p.channels, now);
    store_lanes<V>(p.mixed + static_cast<int64_t>(row) * p.channels + c, acc);
}

// Streamed step, second half: persistent CTAs walk the (sequence, head) pairs.  A producer warp brings a pair's state (one contiguous
// [state][vdim] block) and its x, B and C by bulk copies into one of two stages while the pair before it is worked on; eight warps
// update the state in place and leave the partial outputs; the producer sends the stage's state back and refills it.  vdim and state
// multiples of 4, vdim at most 1024.
constexpr int kStreamThreads = kStepThreads + 32;
struct StreamMeta { float dt, decay, fresh; };
inline size_t ssm_stream_bytes(int state, int vdim) {
    return sizeof(float) * (2 * (static_cast<size_t>(state) * vdim + vdim + 2 * state) + 2 * kStepThreads * 4);
}

__global__ void __launch_bounds__(kStreamThreads) ssm_step_stream_kernel(const SsmParams p, const RowsView rows, int32_t* status) {
    extern __shared__ __align__(16) float sm[];   // 2 x [state * vdim | x: vdim | B: state | C: state], 2 x [threads * 4] partial outputs
    __shared__ uint64_t full[2], done[2];
    __shared__ StreamMeta meta[2];
    __shared__ int gave_up;
    const int P = p.vdim, N = p.state, inner = p.heads * P, block = N * P, stage_floats = block + P + 2 * N, columns = P >> 2,
              slices = kStepThreads / columns;
    const int units = rows.rows * p.heads;
    if (threadIdx.x == 0) {
        for (int s = 0; s < 2; ++s) { mbar_init(&full[s], 1); mbar_init(&done[s], kStepThreads); }
        mbar_fence_init();
        gave_up = 0;
    }
    grid_dependency_wait();
    grid_launch_dependents();
    __syncthreads();

    if (threadIdx.x >= kStepThreads) {   // producer warp; one lane issues, all lanes stay with it
        if ((threadIdx.x & 31) != 0) return;
        float* pending[2] = {nullptr, nullptr};
        int turn = 0;
        for (int unit = blockIdx.x; unit < units + 2 * static_cast<int>(gridDim.x); unit += gridDim.x, ++turn) {
            const int stage = turn & 1, row = unit / p.heads, head = unit - row * p.heads;
            const bool live = unit < units;
            StepRate rate{};
            float* state = nullptr;
            bool fresh = true;
            if (live) {   // operands of this pair, while the stage may still be in use
                const int slot = __ldg(rows.slot + row);
                fresh = rows.lengths[slot] == 0;
                state = p.ssm_state + (static_cast<int64_t>(slot) * p.heads + head) * block;
                rate = step_rate(p, p.projected + static_cast<int64_t>(row) * p.stride, head);
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
            meta[stage] = StreamMeta{rate.dt, rate.decay, fresh ? 1.0f : 0.0f};
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
        const StreamMeta m = meta[stage];
        float* at = sm + stage * stage_floats;
        const float *x = at + block, *B = x + P, *C = B + N;
        float* partial = sm + 2 * stage_floats + stage * kStepThreads * 4;
        float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (active && arrived) {
            float4 xd = *reinterpret_cast<const float4*>(x + column * 4);
            xd = make_float4(xd.x * m.dt, xd.y * m.dt, xd.z * m.dt, xd.w * m.dt);
            float4* s = reinterpret_cast<float4*>(at) + column;
            const bool fresh = m.fresh != 0.0f;
#pragma unroll 4
            for (int n = slice; n < N; n += slices) {
                const float b = B[n], c = C[n];
                float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (!fresh) v = s[n * columns];
                v = make_float4(fmaf(v.x, m.decay, xd.x * b), fmaf(v.y, m.decay, xd.y * b), fmaf(v.z, m.decay, xd.z * b), fmaf(v.w, m.decay, xd.w * b));
                sum = make_float4(fmaf(v.x, c, sum.x), fmaf(v.y, c, sum.y), fmaf(v.z, c, sum.z), fmaf(v.w, c, sum.w));
                s[n * columns] = v;
            }
        }
        reinterpret_cast<float4*>(partial)[threadIdx.x] = sum;
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // the updated state is read by the copy engine
        asm volatile("bar.sync 1, %0;" ::"n"(kStepThreads) : "memory");
        if (*static_cast<volatile int*>(&gave_up)) return;   // a state never arrived: the eight warps leave together
        for (int i = threadIdx.x; i < P; i += kStepThreads) {
            float total = 0.0f;
            for (int k = 0; k < slices; ++k) total += partial[k * P + i];
            p.y[static_cast<int64_t>(row) * inner + head * P + i] = fmaf(skip_of(p, head), x[i], total);
        }
        mbar_arrive(&done[stage]);
    }
}

// grid (heads, sequences); one row per sequence.  V = 4 when vdim is a multiple of 4.
template <int V>
__global__ void __launch_bounds__(kStepThreads, 4) ssm_step_kernel(const SsmParams p, const RowsView rows) {
    extern __shared__ __align__(16) float sm[];   // [vdim + 2 state] convolved channels, then [threads * V] partial outputs
    const int P = p.vdim, N = p.state, head = blockIdx.x, row = blockIdx.y;
    const int inner = p.heads * P;
    float* mixed = sm;
    float* partial = sm + ((P + 2 * N + 3) & ~3);
    grid_dependency_wait();
    grid_launch_dependents();
    const int slot = __ldg(rows.slot + row);   // one row per sequence: row and sequence are the same number
    const RowPlace place{row, slot, rows.lengths[slot]};
    const float* in = p.projected + static_cast<int64_t>(row) * p.stride;
    const bool fresh = place.position == 0;
    float* state = p.ssm_state + (static_cast<int64_t>(place.slot) * p.heads + head) * N * P;

    // this thread's part of the state: value columns p0.., every `slices`-th state row; the first batch is requested before
    // the convolution so that its latency is covered
    const int columns = P / V, slices = kStepThreads / columns > 0 ? kStepThreads / columns : 1;
    constexpr int kAhead = 8;
    const int my_slice = columns <= kStepThreads ? static_cast<int>(threadIdx.x) / columns : 0;
    const int my_column = static_cast<int>(threadIdx.x) - my_slice * columns;
    auto fetch = [&](Lanes<V>(&s)[kAhead], int n0, int column, bool active) {
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int n = n0 + i * slices;
#pragma unroll
            for (int k = 0; k < V; ++k) s[i].v[k] = 0.0f;
            if (active && !fresh && n < N) s[i] = load_lanes<V>(state + static_cast<int64_t>(n) * P + column * V);
        }
    };
    Lanes<V> s[kAhead];
    fetch(s, my_slice, my_column, my_column < columns && my_slice < slices);

    convolve_head(p, in, place.slot, place.position, head, mixed);
    const auto [dt, decay] = step_rate(p, in, head);
    __syncthreads();
    const float *x = mixed, *B = mixed + P, *C = mixed + P + N;

    for (int base = 0; base < columns; base += kStepThreads) {
        const int column = base + my_column, slice = my_slice;
        const bool active = column < columns && slice < slices;
        Lanes<V> sum;
#pragma unroll
        for (int k = 0; k < V; ++k) sum.v[k] = 0.0f;
        if (active) {
            Lanes<V> xd;
#pragma unroll
            for (int k = 0; k < V; ++k) xd.v[k] = x[column * V + k] * dt;
            for (int n0 = slice; n0 < N; n0 += slices * kAhead) {
                if (base > 0 || n0 != slice) fetch(s, n0, column, true);
#pragma unroll
                for (int i = 0; i < kAhead; ++i) {
                    const int n = n0 + i * slices;
                    if (n >= N) continue;
                    const float b = B[n], c = C[n];
#pragma unroll
                    for (int k = 0; k < V; ++k) {
                        s[i].v[k] = fmaf(s[i].v[k], decay, xd.v[k] * b);
                        sum.v[k] = fmaf(s[i].v[k], c, sum.v[k]);
                    }
                    store_lanes<V>(state + static_cast<int64_t>(n) * P + column * V, s[i]);
                }
            }
        }
        __syncthreads();
        store_lanes<V>(partial + threadIdx.x * V, sum);
        __syncthreads();
        const int width = columns <= kStepThreads ? columns : min(kStepThreads, columns - base);
        for (int i = threadIdx.x; i < width * V; i += kStepThreads) {
            float total = 0.0f;
            for (int s = 0; s < slices; ++s) total += partial[(s * (columns <= kStepThreads ? columns : 0)) * V + i];
            const int at = base * V + i;
            p.y[static_cast<int64_t>(row) * inner + head * P + at] = fmaf(skip_of(p, head), x[at], total);
        }
    }
}

// mixed[row, c] = silu(conv(x | B | C)), grid (channel blocks, strips of kConvRows rows).  V channels per thread (4 when rows and
// channel counts allow 16-byte accesses).  TAPS > 0: the inputs of a strip slide through registers, each read once; TAPS = 0: any
// number of taps, read from L1 again.
constexpr int kConvRows = 16;
template <int V, int TAPS> __global__ void __launch_bounds__(128) short_conv_kernel(const SsmParams p, const RowsView rows) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V, inner = p.heads * p.vdim;
    if (c >= p.channels) return;
    const int row0 = blockIdx.y * kConvRows, row1 = min(rows.rows, row0 + kConvRows);
    // input of the token `back` places before `row`
    auto input = [&](int row, int offset, const RowPlace& place, int back) {
        if (back <= offset) return load_lanes<V>(p.projected + static_cast<int64_t>(row - back) * p.stride + inner + c);
        Lanes<V> old;
#pragma unroll
        for (int k = 0; k < V; ++k) old.v[k] = ring_input(p, place.slot, place.position - back, c + k);
        return old;
    };
    const Lanes<V> bias = load_lanes<V>(p.conv_bias + c);
    Lanes<V> weight[TAPS > 0 ? TAPS : 1], window[TAPS > 0 ? TAPS : 1];
    if constexpr (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
            for (int k = 0; k < V; ++k) weight[j].v[k] = p.conv_weight[static_cast<int64_t>(c + k) * TAPS + j];
    }
    int sequence = -1;
    for (int row = row0; row < row1; ++row) {
        const RowPlace place = row_place(rows, row);
        const int offset = row - __ldg(rows.first + place.sequence);
        Lanes<V> acc = bias;
        if constexpr (TAPS > 0) {
            if (place.sequence != sequence) {   // the strip enters a sequence: its earlier inputs
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) window[j] = input(row, offset, place, TAPS - 1 - j);
                sequence = place.sequence;
            }
            window[TAPS - 1] = input(row, offset, place, 0);
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
#pragma unroll
                for (int k = 0; k < V; ++k) acc.v[k] = fmaf(weight[j].v[k], window[j].v[k], acc.v[k]);
#pragma unroll
            for (int j = 0; j + 1 < TAPS; ++j) window[j] = window[j + 1];
        } else {
            for (int j = 0; j < p.taps; ++j) {
                const Lanes<V> v = input(row, offset, place, p.taps - 1 - j);
#pragma unroll
                for (int k = 0; k < V; ++k) acc.v[k] = fmaf(p.conv_weight[static_cast<int64_t>(c + k) * p.taps + j], v.v[k], acc.v[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < V; ++k) acc.v[k] *= sigmoid_exact(acc.v[k]);
        store_lanes<V>(p.mixed + static_cast<int64_t>(row) * p.channels + c, acc);
    }
}
template <int V, int TAPS> int launch_conv(const SsmParams& p, const RowsView& rows, cudaStream_t stream) {
    const dim3 grid(static_cast<unsigned>((p.channels / V + 127) / 128), static_cast<unsigned>((rows.rows + kConvRows - 1) / kConvRows));
    return cuda_status(launch_dependent(short_conv_kernel<V, TAPS>, grid, dim3(128), 0, stream, p, rows), "short_conv_kernel launch");
}
template <int V> int pick_conv(const SsmParams& p, const RowsView& rows, cudaStream_t stream) {
    switch (p.taps) {
    case 2: return launch_conv<V, 2>(p, rows, stream);
    case 3: return launch_conv<V, 3>(p, rows, stream);
    case 4: return launch_conv<V, 4>(p, rows, stream);
    }
    return launch_conv<V, 0>(p, rows, stream);
}

// The last inputs of every sequence into its slot's ring, grid (channel blocks, sequences)
__global__ void __launch_bounds__(256) conv_ring_kernel(const SsmParams p, const RowsView rows) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
    if (c >= p.channels) return;
    const int first = __ldg(rows.first + s), count = __ldg(rows.first + s + 1) - first, slot = __ldg(rows.slot + s);
    const int length = rows.lengths[slot], inner = p.heads * p.vdim;
    for (int t = max(0, count - p.taps); t < count; ++t)
        p.conv_state[(static_cast<int64_t>(slot) * p.taps + (length + t) % p.taps) * p.channels + c] =
            p.projected[static_cast<int64_t>(first + t) * p.stride + inner + c];
}

// ---- scan -----------------------------------------------------------------------------------------------------
constexpr int kScanWarps = 4;

// LN lanes of a warp share the state dimension (4 * Q values each, in quads LN * 4 apart), the other 32 / LN lane groups hold
// four value columns each.  grid (column tiles, heads, sequences).
template <int LN, int Q>
__global__ void __launch_bounds__(kScanWarps * 32, LN * Q <= 32 ? 4 : 3) ssm_scan_kernel(const SsmParams p, const RowsView rows) {
    constexpr int kNp = LN * 4 * Q;                      // padded state size
    constexpr int kScanTokens = kNp <= 128 ? 16 : 4;     // tokens staged at a time
    constexpr int kGroups = 32 / LN;
    constexpr int kColumns = kScanWarps * kGroups * 4;   // value columns of the CTA
    __shared__ __align__(16) float sB[2][kScanTokens][kNp], sC[2][kScanTokens][kNp], sx[2][kScanTokens][kColumns];
    __shared__ float sdt[2][kScanTokens];
    grid_dependency_wait();
    grid_launch_dependents();
    const int P = p.vdim, N = p.state, head = blockIdx.y, s = blockIdx.z, column0 = blockIdx.x * kColumns;
    const int group = head / (p.heads / p.groups), inner = p.heads * P;
    const int first = __ldg(rows.first + s), count = __ldg(rows.first + s + 1) - first, slot = __ldg(rows.slot + s);
    const bool fresh = rows.lengths[slot] == 0;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ln = lane % LN, lg = lane / LN;
    const int local = (warp * kGroups + lg) * 4;         // first of this lane's four value columns inside the tile
    const int column = column0 + local;
    float* state = p.ssm_state + (static_cast<int64_t>(slot) * p.heads + head) * N * P;

    for (int i = threadIdx.x; i < 2 * kScanTokens * kNp; i += blockDim.x) { (&sB[0][0][0])[i] = 0.0f; (&sC[0][0][0])[i] = 0.0f; }
    for (int i = threadIdx.x; i < 2 * kScanTokens * kColumns; i += blockDim.x) (&sx[0][0][0])[i] = 0.0f;
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
    const bool fixed = p.fixed_decay != nullptr;
    const float rate = fixed ? p.fixed_decay[head] : -expf(p.a_log[head]), dt_bias = fixed ? 0.0f : p.dt_bias[head], skip = skip_of(p, head);
    const int live_columns = min(kColumns, P - column0);
    const bool aligned = ((p.channels | P | N | inner) & 3) == 0 && (reinterpret_cast<uintptr_t>(p.mixed) & 15) == 0;

    auto stage = [&](int chunk) {
        const int buffer = chunk & 1, t0 = chunk * kScanTokens, tokens = min(kScanTokens, count - t0);
        // a warp per token; 16 bytes per copy where every row and slice starts on such a boundary
        const float* from[3] = {p.mixed + head * P + column0, p.mixed + inner + group * N, p.mixed + inner + (p.groups + group) * N};
        const int width[3] = {live_columns, N, N};
        for (int t = warp; t < tokens; t += kScanWarps) {
            const int64_t row = static_cast<int64_t>(first + t0 + t) * p.channels;
            float* to[3] = {sx[buffer][t], sB[buffer][t], sC[buffer][t]};
#pragma unroll
            for (int part = 0; part < 3; ++part) {
                if (aligned) {
                    for (int c = lane * 4; c < width[part]; c += 128) copy_async_16(smem_u32(to[part] + c), from[part] + row + c, true);
                } else {
                    for (int c = lane; c < width[part]; c += 32) copy_async_4(to[part] + c, from[part] + row + c);
                }
            }
        }
        if (!fixed && threadIdx.x < tokens)
            copy_async_4(&sdt[buffer][threadIdx.x], p.projected + static_cast<int64_t>(first + t0 + threadIdx.x) * p.stride + inner + p.channels + head);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    const int chunks = (count + kScanTokens - 1) / kScanTokens;
    // after the exchanges below a lane holds column `mine` of its four, summed; lanes ln < 4 write
    const bool odd = lane & 1, second = lane & 2;
    const int mine = (odd ? 2 : 0) + (second ? 1 : 0);
    const bool writes = ln < 4 && column + mine < P;
    stage(0);
    for (int chunk = 0; chunk < chunks; ++chunk) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                  // the chunk has landed; the other buffer is free
        if (chunk + 1 < chunks) stage(chunk + 1);
        const int buffer = chunk & 1, t0 = chunk * kScanTokens, tokens = min(kScanTokens, count - t0);
        // step size and decay of token `lane` of the chunk, handed round by shuffles
        float dt_mine = 1.0f, decay_mine = rate;
        if (!fixed && lane < tokens) {
            dt_mine = softplus(sdt[buffer][lane] + dt_bias);
            decay_mine = expf(rate * dt_mine);
        }
        float* const y_chunk = p.y + static_cast<int64_t>(first + t0) * inner + head * P + column + mine;
        auto token = [&](int t) {
            const float dt = __shfl_sync(0xffffffffu, dt_mine, t), decay = __shfl_sync(0xffffffffu, decay_mine, t);
            const float4 xv = *reinterpret_cast<const float4*>(&sx[buffer][t][local]);
            const float x[4] = {xv.x, xv.y, xv.z, xv.w};
            const uint64_t decay2 = pack2(decay, decay);
            uint64_t xd[4], acc[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) xd[k] = pack2(x[k] * dt, x[k] * dt);
#pragma unroll
            for (int q = 0; q < Q; ++q) {
                const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(&sB[buffer][t][q * LN * 4 + ln * 4]);
                const ulonglong2 c = *reinterpret_cast<const ulonglong2*>(&sC[buffer][t][q * LN * 4 + ln * 4]);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    S[k][2 * q] = fma2(S[k][2 * q], decay2, mul2(xd[k], b.x));
                    acc[k] = q == 0 ? mul2(S[k][0], c.x) : fma2(S[k][2 * q], c.x, acc[k]);
                    S[k][2 * q + 1] = fma2(S[k][2 * q + 1], decay2, mul2(xd[k], b.y));
                    acc[k] = fma2(S[k][2 * q + 1], c.y, acc[k]);
                }
            }
            float part[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) { const float2 v = unpack2(acc[k]); part[k] = v.x + v.y; }
            // sum over the LN lanes: two exchanges halve the four columns, the rest are plain butterflies
            const float keep0 = odd ? part[2] : part[0], give0 = odd ? part[0] : part[2];
            const float keep1 = odd ? part[3] : part[1], give1 = odd ? part[1] : part[3];
            const float two0 = keep0 + __shfl_xor_sync(0xffffffffu, give0, 1), two1 = keep1 + __shfl_xor_sync(0xffffffffu, give1, 1);
            float one = (second ? two1 : two0) + __shfl_xor_sync(0xffffffffu, second ? two0 : two1, 2);
#pragma unroll
            for (int o = 4; o < LN; o <<= 1) one += __shfl_xor_sync(0xffffffffu, one, o);
            if (writes) y_chunk[static_cast<int64_t>(t) * inner] = fmaf(skip, sx[buffer][t][local + mine], one);
        };
        if (tokens == kScanTokens) {
#pragma unroll 4
            for (int t = 0; t < kScanTokens; ++t) token(t);
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
    constexpr int kColumns = kScanWarps * (32 / LN) * 4;
    const dim3 grid(static_cast<unsigned>((p.vdim + kColumns - 1) / kColumns), static_cast<unsigned>(p.heads), static_cast<unsigned>(rows.sequences));
    return cuda_status(launch_dependent(ssm_scan_kernel<LN, Q>, grid, dim3(kScanWarps * 32), 0, stream, p, rows), "ssm_scan_kernel launch");
}

// grid (rows, parts).  V adjacent values per access (4 when everything allows 16-byte accesses).  GATE_FIRST: the norm of y * silu(z);
// otherwise the norm of y, times sigmoid(z) * factor.
template <int V, bool GATE_FIRST>
__global__ void __launch_bounds__(128) gated_group_norm_kernel(const float* y, const float* z, int64_t z_stride, const float* weight, int width,
                                                               int parts, float eps, float factor, float* out, __nv_bfloat16* out_hi,
                                                               __nv_bfloat16* out_lo, int64_t out_stride) {
    __shared__ float scratch[32];
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    const int size = width / parts, c0 = blockIdx.y * size;
    constexpr int kKeep = 4;   // accesses whose values a thread keeps in registers; longer parts are computed again
    Lanes<V> kept[kKeep];
    float squares = 0.0f;
    auto value = [&](int c) {
        Lanes<V> v = load_lanes<V>(y + row * width + c0 + c);
        if constexpr (GATE_FIRST) {
            const Lanes<V> g = load_lanes<V>(z + row * z_stride + c0 + c);
#pragma unroll
            for (int k = 0; k < V; ++k) v.v[k] *= g.v[k] * sigmoid_exact(g.v[k]);
        }
        return v;
    };
    auto finish = [&](int c, const Lanes<V>& v, float inverse) {
        const Lanes<V> w = load_lanes<V>(weight + c0 + c);
        Lanes<V> r;
#pragma unroll
        for (int k = 0; k < V; ++k) r.v[k] = v.v[k] * inverse * w.v[k];
        if constexpr (!GATE_FIRST) {
            const Lanes<V> g = load_lanes<V>(z + row * z_stride + c0 + c);
#pragma unroll
            for (int k = 0; k < V; ++k) r.v[k] *= sigmoid_exact(g.v[k]) * factor;
        }
        const int64_t at = row * out_stride + c0 + c;
        if constexpr (V == 4) {
            if (out) store_lanes<V>(out + at, r);
            if (out_hi) {
                uint2 hi, lo;
                pack_planes(r.v[0], r.v[1], hi.x, lo.x);
                pack_planes(r.v[2], r.v[3], hi.y, lo.y);
                *reinterpret_cast<uint2*>(out_hi + at) = hi;
                if (out_lo) *reinterpret_cast<uint2*>(out_lo + at) = lo;
            }
        } else {
            store_forms(r.v[0], at, out, out_hi, out_lo);
        }
    };
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
        const int c = (threadIdx.x + i * 128) * V;
        if (c < size) kept[i] = value(c);
#pragma unroll
        for (int k = 0; k < V; ++k) squares = c < size ? fmaf(kept[i].v[k], kept[i].v[k], squares) : squares;
    }
    for (int c = (threadIdx.x + kKeep * 128) * V; c < size; c += 128 * V) {
        const Lanes<V> v = value(c);
#pragma unroll
        for (int k = 0; k < V; ++k) squares = fmaf(v.v[k], v.v[k], squares);
    }
    squares = block_sum(squares, scratch);
    const float inverse = 1.0f / sqrtf(squares / static_cast<float>(size) + eps);
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
        const int c = (threadIdx.x + i * 128) * V;
        if (c < size) finish(c, kept[i], inverse);
    }
    for (int c = (threadIdx.x + kKeep * 128) * V; c < size; c += 128 * V) finish(c, value(c), inverse);
}

template <bool GATE_FIRST>
int launch_group_norm(const float* y, const float* z, int64_t z_stride, const float* weight, int64_t rows, int64_t width, int32_t parts, double eps,
                      float factor, float* out, void* out_hi, void* out_lo, int64_t out_stride, void* stream, const char* what) {
    if (!y || !z || !weight || rows < 0 || width <= 0 || width > INT32_MAX || parts <= 0 || width % parts || parts > 65535 || (!out && !out_hi)
        || out_stride < width) {
        set_error("%s: bad pointer or size", what);
        return B200_BAD_ARGUMENT;
    }
    if (rows == 0) return B200_OK;
    const bool quads = (width / parts) % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0
        && ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(out)
             | (reinterpret_cast<uintptr_t>(out_hi) << 1) | (reinterpret_cast<uintptr_t>(out_lo) << 1)) & 15) == 0;
    return cuda_status(launch_dependent(quads ? gated_group_norm_kernel<4, GATE_FIRST> : gated_group_norm_kernel<1, GATE_FIRST>,
                                        dim3(static_cast<unsigned>(rows), static_cast<unsigned>(parts)), dim3(128), 0, as_stream(stream), y, z, z_stride,
                                        weight, static_cast<int>(width), static_cast<int>(parts), static_cast<float>(eps), factor, out,
                                        static_cast<__nv_bfloat16*>(out_hi), static_cast<__nv_bfloat16*>(out_lo), out_stride),
                       "gated_group_norm_kernel launch");
}

// An RMS norm per head of `size` values, times weight [size], times silu(z): a warp per (row, head), the head in registers.  V adjacent
// values per access.
constexpr int kHeadNormWarps = 8, kHeadNormKeep = 4;
template <int V>
__global__ void __launch_bounds__(kHeadNormWarps * 32) head_norm_gated_kernel(const float* y, const float* z, int64_t z_stride, const float* weight, int64_t units,
                                                                             int heads, int size, float eps, float* out, __nv_bfloat16* out_hi,
                                                                             __nv_bfloat16* out_lo, int64_t out_stride) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t unit = static_cast<int64_t>(blockIdx.x) * kHeadNormWarps + (threadIdx.x >> 5);
    if (unit >= units) return;
    const int lane = threadIdx.x & 31;
    const int64_t row = unit / heads;
    const int head = static_cast<int>(unit - row * heads);
    const float *from = y + unit * size, *gate = z + row * z_stride + static_cast<int64_t>(head) * size;
    const int64_t to = row * out_stride + static_cast<int64_t>(head) * size;
    Lanes<V> kept[kHeadNormKeep];
    float squares = 0.0f;
    auto add = [&](const Lanes<V>& v) {
#pragma unroll
        for (int k = 0; k < V; ++k) squares = fmaf(v.v[k], v.v[k], squares);
    };
#pragma unroll
    for (int i = 0; i < kHeadNormKeep; ++i) {
        const int c = (lane + i * 32) * V;
        if (c < size) { kept[i] = load_lanes<V>(from + c); add(kept[i]); }
    }
    for (int c = (lane + kHeadNormKeep * 32) * V; c < size; c += 32 * V) add(load_lanes<V>(from + c));
    const float inverse = 1.0f / sqrtf(warp_sum(squares) / static_cast<float>(size) + eps);
    auto finish = [&](int c, Lanes<V> v) {
        const Lanes<V> w = load_lanes<V>(weight + c), g = load_lanes<V>(gate + c);
#pragma unroll
        for (int k = 0; k < V; ++k) v.v[k] = v.v[k] * inverse * w.v[k] * (g.v[k] * sigmoid_exact(g.v[k]));
        if constexpr (V == 4) {
            if (out) store_lanes<V>(out + to + c, v);
            if (out_hi) {
                uint2 hi, lo;
                pack_planes(v.v[0], v.v[1], hi.x, lo.x);
                pack_planes(v.v[2], v.v[3], hi.y, lo.y);
                *reinterpret_cast<uint2*>(out_hi + to + c) = hi;
                if (out_lo) *reinterpret_cast<uint2*>(out_lo + to + c) = lo;
            }
        } else {
            store_forms(v.v[0], to + c, out, out_hi, out_lo);
        }
    };
#pragma unroll
    for (int i = 0; i < kHeadNormKeep; ++i) {
        const int c = (lane + i * 32) * V;
        if (c < size) finish(c, kept[i]);
    }
    for (int c = (lane + kHeadNormKeep * 32) * V; c < size; c += 32 * V) finish(c, load_lanes<V>(from + c));
}

__global__ void rows_advance_kernel(const RowsView rows, const int64_t* ids, int32_t* last) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int s = blockIdx.x * blockDim.x + threadIdx.x;
    if (s >= rows.sequences) return;
    rows.lengths[rows.slot[s]] += rows.first[s + 1] - rows.first[s];
    if (last) last[rows.slot[s]] = static_cast<int32_t>(ids[rows.first[s + 1] - 1]);
}

__global__ void __launch_bounds__(256) dynamic_tanh_kernel(const float* x, const float* add_rows, const float* add_vector, int width,
                                                           b200_elementwise_norm norm, float* sum, float* out, __nv_bfloat16* out_hi,
                                                           __nv_bfloat16* out_lo) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < width; c += gridDim.y * blockDim.x) {
        const int64_t at = row * width + c;
        float v = x[at];
        if (add_rows) v += add_rows[at];
        if (add_vector) v += add_vector[c];
        if (sum) sum[at] = v;
        store_forms(fmaf(tanhf(norm.alpha * v), norm.weight[c], norm.bias[c]), at, out, out_hi, out_lo);
    }
}

template <class T>
__global__ void __launch_bounds__(256) embedding_scaled_kernel(const T* table, const int64_t* ids, int64_t vocab, int64_t width, float scale,
                                                               float* out, int32_t* status) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    int64_t id = ids[row];
    if (id < 0 || id >= vocab) {   // the host API validates ids it can see; device-resident ids are clamped and flagged
        if (threadIdx.x == 0) atomicExch(status, B200_BAD_ARGUMENT);
        id = id < 0 ? 0 : vocab - 1;
    }
    for (int64_t c = threadIdx.x; c < width; c += blockDim.x) out[row * width + c] = load_as_f32(table, id * width + c) * scale;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_rows_advance(const b200_rows* pass, void* stream) {
    RowsView rows;
    if (!rows_view(pass, rows)) return B200_BAD_ARGUMENT;
    return cuda_status(launch_dependent(rows_advance_kernel, dim3((rows.sequences + 127) / 128), dim3(128), 0, as_stream(stream), rows,
                                        static_cast<const int64_t*>(nullptr), static_cast<int32_t*>(nullptr)), "rows_advance_kernel launch");
}

int b200_rows_advance_tokens(const b200_rows* pass, const int64_t* ids, int32_t* last, void* stream) {
    RowsView rows;
    if (!rows_view(pass, rows)) return B200_BAD_ARGUMENT;
    if (!ids || !last) { set_error("b200_rows_advance_tokens: bad pointer"); return B200_BAD_ARGUMENT; }
    return cuda_status(launch_dependent(rows_advance_kernel, dim3((rows.sequences + 127) / 128), dim3(128), 0, as_stream(stream), rows, ids, last),
                       "rows_advance_kernel launch");
}

int b200_embedding_scaled(const void* table, int32_t table_dtype, const int64_t* ids, int64_t rows, int64_t vocab, int64_t width, float scale,
                          float* out, void* stream) {
    if (!table || !ids || !out || rows < 0 || vocab <= 0 || width <= 0) { set_error("b200_embedding_scaled: bad pointer or size"); return B200_BAD_ARGUMENT; }
    if (rows == 0) return B200_OK;
    int device = 0;
    B200_CUDA(cudaGetDevice(&device));
    int32_t* status = device_status_word(device);
    if (!status) { set_error("b200_embedding_scaled: the device status word could not be allocated"); return B200_NO_DEVICE; }
    const dim3 grid(static_cast<unsigned>(rows));
    if (table_dtype == B200_BF16)
        return cuda_status(launch_dependent(embedding_scaled_kernel<__nv_bfloat16>, grid, dim3(256), 0, as_stream(stream),
                                            static_cast<const __nv_bfloat16*>(table), ids, vocab, width, scale, out, status), "embedding_scaled_kernel launch");
    if (table_dtype == B200_F32)
        return cuda_status(launch_dependent(embedding_scaled_kernel<float>, grid, dim3(256), 0, as_stream(stream), static_cast<const float*>(table),
                                            ids, vocab, width, scale, out, status), "embedding_scaled_kernel launch");
    set_error("b200_embedding_scaled: table dtype %d is not f32 or bf16", table_dtype);
    return B200_UNSUPPORTED;
}

int b200_dynamic_tanh(const float* x, const float* add_rows, const float* add_vector, int64_t rows, int64_t width,
                      const b200_elementwise_norm* norm, float* sum, float* out, void* out_hi, void* out_lo, void* stream) {
    if (!x || !norm || !norm->weight || !norm->bias || rows < 0 || width <= 0 || width > INT32_MAX || (!out && !out_hi)) {
        set_error("b200_dynamic_tanh: bad pointer or size");
        return B200_BAD_ARGUMENT;
    }
    if (rows == 0) return B200_OK;
    const unsigned slices = static_cast<unsigned>(rows >= 512 ? 1 : (width + 1023) / 1024);
    return cuda_status(launch_dependent(dynamic_tanh_kernel, dim3(static_cast<unsigned>(rows), slices), dim3(256), 0, as_stream(stream), x, add_rows,
                                        add_vector, static_cast<int>(width), *norm, sum, out, static_cast<__nv_bfloat16*>(out_hi),
                                        static_cast<__nv_bfloat16*>(out_lo)), "dynamic_tanh_kernel launch");
}

int b200_ssm_forward(const b200_ssm_args* a, const b200_rows* pass, void* stream) {
    RowsView rows;
    if (!rows_view(pass, rows)) return B200_BAD_ARGUMENT;
    const int rates = !a || a->decay ? 0 : a->delta ? 2 : 1;   // columns per head behind the channels
    if (!a || a->heads <= 0 || a->vdim <= 0 || a->state <= 0 || a->groups <= 0 || a->heads % a->groups || a->taps <= 0
        || (a->conv_weight ? !a->conv_bias || !a->conv_state : a->taps != 1) || (!a->decay && (!a->dt_bias || !a->a_log || (!a->d && !a->delta))) || !a->ssm_state
        || (a->delta && (a->decay || !a->conv_weight))
        || !a->projected || !a->y || (a->stride && a->stride < 2 * int64_t{a->heads} * a->vdim + 2 * int64_t{a->groups} * a->state + rates * a->heads)
        || a->stride > INT32_MAX) {
        set_error("b200_ssm_forward: bad pointer or size");
        return B200_BAD_ARGUMENT;
    }
    SsmParams p{};
    p.heads = a->heads; p.vdim = a->vdim; p.state = a->state; p.groups = a->groups; p.taps = a->taps;
    p.channels = a->heads * a->vdim + 2 * a->groups * a->state;
    p.stride = a->stride ? static_cast<int>(a->stride) : a->heads * a->vdim + p.channels + rates * a->heads;
    p.fixed_decay = a->decay;
    p.conv_weight = a->conv_weight; p.conv_bias = a->conv_bias; p.dt_bias = a->dt_bias; p.a_log = a->a_log; p.d = a->d;
    p.conv_state = a->conv_state; p.ssm_state = a->ssm_state; p.projected = a->projected; p.mixed = a->mixed; p.y = a->y;
    cudaStream_t s = as_stream(stream);
    if (rows.max_count == 1) {
        const bool quads = a->vdim % 4 == 0 && (reinterpret_cast<uintptr_t>(a->ssm_state) & 15) == 0;
        const size_t streamed = a->delta ? 0 : ssm_stream_bytes(a->state, a->vdim);
        const bool aligned = ((reinterpret_cast<uintptr_t>(p.projected) | reinterpret_cast<uintptr_t>(p.mixed) | reinterpret_cast<uintptr_t>(p.conv_bias)
                               | reinterpret_cast<uintptr_t>(p.conv_state)) & 15) == 0;
        int device = 0;
        B200_CUDA(cudaGetDevice(&device));
        const int64_t units = static_cast<int64_t>(rows.rows) * a->heads;
        const int64_t per_sm = std::min<int64_t>(7, (228 * 1024) / (streamed + 1024 + 128)), resident = sm_count(device) * per_sm;
        // streaming pays from a few pairs per CTA on; below that its extra launch and ramp cost more
        const bool streams = a->mixed && aligned
            && (a->delta ? delta_step_streams(p, rows, sm_count(device))
                         : quads && a->state % 4 == 0 && a->vdim <= 4 * kStepThreads && streamed <= 110 * 1024 && units >= 4 * resident);
        if (streams) {
            int32_t* status = device_status_word(device);
            if (!status) { set_error("the device status word could not be allocated"); return B200_NO_DEVICE; }
            auto stream_steps = [&]() -> int {
                if (a->delta) return launch_delta_step_stream(p, rows, sm_count(device), status, s);
                B200_CUDA(cudaFuncSetAttribute(ssm_step_stream_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(streamed)));
                return cuda_status(launch_dependent(ssm_step_stream_kernel, dim3(static_cast<unsigned>(std::min(units, resident))), dim3(kStreamThreads), streamed, s, p, rows,
                                                    status), "ssm_step_stream_kernel launch");
            };
            // (rows of `projected` start on 16-byte boundaries only when their stride is a multiple of 4)
            const unsigned quads_per_row = static_cast<unsigned>(p.stride % 4 == 0 ? 4 : 1);
            if (!p.conv_weight) {
                const int activated = quads_per_row == 4 ? launch_activate<4>(p, rows.rows, s) : launch_activate<1>(p, rows.rows, s);
                if (activated != B200_OK) return activated;
                return stream_steps();
            }
            const dim3 grid((static_cast<unsigned>(p.channels) / quads_per_row + 127) / 128, static_cast<unsigned>(rows.rows));
            const int conv = cuda_status(launch_dependent(quads_per_row == 4 ? conv_step_kernel<4> : conv_step_kernel<1>, grid, dim3(128), 0, s, p, rows),
                                         "conv_step_kernel launch");
            return conv != B200_OK ? conv : stream_steps();
        }
        if (a->delta) return launch_delta_step(p, rows, s);
        const size_t smem = sizeof(float) * (((a->vdim + 2 * a->state + 3) & ~3) + kStepThreads * (quads ? 4 : 1));
        if (smem > 200 * 1024) { set_error("b200_ssm_forward: a head of %d x %d values does not fit shared memory", a->state, a->vdim); return B200_UNSUPPORTED; }
        auto kernel = quads ? ssm_step_kernel<4> : ssm_step_kernel<1>;
        if (smem > 46 * 1024) B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        return cuda_status(launch_dependent(kernel, dim3(static_cast<unsigned>(a->heads), static_cast<unsigned>(rows.sequences)), dim3(kStepThreads),
                                            smem, s, p, rows), "ssm_step_kernel launch");
    }
    if (!a->mixed) { set_error("b200_ssm_forward: workspace missing"); return B200_BAD_ARGUMENT; }
    if (a->state > B200_SSM_MAX_STATE) { set_error("b200_ssm_forward: state sizes above %d are not supported", B200_SSM_MAX_STATE); return B200_UNSUPPORTED; }
    if (rows.sequences > 65535) { set_error("b200_ssm_forward: too many sequences in one pass"); return B200_UNSUPPORTED; }
    const unsigned blocks = static_cast<unsigned>((p.channels + 255) / 256);
    const bool conv_quads = p.channels % 4 == 0 && p.stride % 4 == 0 && (p.heads * p.vdim) % 4 == 0
        && ((reinterpret_cast<uintptr_t>(p.projected) | reinterpret_cast<uintptr_t>(p.mixed) | reinterpret_cast<uintptr_t>(p.conv_bias)) & 15) == 0;
    int status = B200_OK;
    if (!p.conv_weight) {
        if (rows.rows > 65535) { set_error("b200_ssm_forward: at most 65535 rows in one pass"); return B200_UNSUPPORTED; }
        status = conv_quads ? launch_activate<4>(p, rows.rows, s) : launch_activate<1>(p, rows.rows, s);
    } else {
        status = conv_quads ? pick_conv<4>(p, rows, s) : pick_conv<1>(p, rows, s);
        if (status != B200_OK) return status;
        status = cuda_status(launch_dependent(conv_ring_kernel, dim3(blocks, static_cast<unsigned>(rows.sequences)), dim3(256), 0, s, p, rows), "conv_ring_kernel launch");
    }
    if (status != B200_OK) return status;
    if (a->delta) return launch_delta_scan(p, rows, s);
    if (a->state <= 32) return launch_scan<8, 1>(p, rows, s);
    if (a->state <= 64) return launch_scan<8, 2>(p, rows, s);
    if (a->state <= 96) return launch_scan<8, 3>(p, rows, s);
    if (a->state <= 128) return launch_scan<8, 4>(p, rows, s);
    if (a->state <= 256) return launch_scan<32, 2>(p, rows, s);
    return launch_scan<32, 4>(p, rows, s);
}

int b200_gated_group_norm(const float* y, const float* z, int64_t z_stride, const float* weight, int64_t rows, int64_t width, int32_t parts,
                          double eps, float* out, void* out_hi, void* out_lo, void* stream) {
    return launch_group_norm<true>(y, z, z_stride, weight, rows, width, parts, eps, 1.0f, out, out_hi, out_lo, width, stream, "b200_gated_group_norm");
}

int b200_norm_gated(const float* y, const float* gate, int64_t gate_stride, const float* weight, int64_t rows, int64_t width, int32_t parts, double eps,
                    float factor, float* out, void* out_hi, void* out_lo, int64_t out_stride, void* stream) {
    return launch_group_norm<false>(y, gate, gate_stride, weight, rows, width, parts, eps, factor, out, out_hi, out_lo, out_stride, stream, "b200_norm_gated");
}

int b200_head_norm_gated(const float* y, const float* gate, int64_t gate_stride, const float* weight, int64_t rows, int32_t heads, int32_t size, double eps,
                         float* out, void* out_hi, void* out_lo, int64_t out_stride, void* stream) {
    if (!y || !gate || !weight || rows < 0 || heads <= 0 || size <= 0 || (!out && !out_hi) || out_stride < static_cast<int64_t>(heads) * size
        || rows * heads > int64_t{INT32_MAX} * kHeadNormWarps) {
        set_error("b200_head_norm_gated: bad pointer or size");
        return B200_BAD_ARGUMENT;
    }
    if (rows == 0) return B200_OK;
    const bool quads = size % 4 == 0 && gate_stride % 4 == 0 && out_stride % 4 == 0
        && ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(out)
             | (reinterpret_cast<uintptr_t>(out_hi) << 1) | (reinterpret_cast<uintptr_t>(out_lo) << 1)) & 15) == 0;
    const int64_t units = rows * heads;
    return cuda_status(launch_dependent(quads ? head_norm_gated_kernel<4> : head_norm_gated_kernel<1>,
                                        dim3(static_cast<unsigned>((units + kHeadNormWarps - 1) / kHeadNormWarps)), dim3(kHeadNormWarps * 32), 0, as_stream(stream), y,
                                        gate, gate_stride, weight, units, static_cast<int>(heads), static_cast<int>(size), static_cast<float>(eps), out,
                                        static_cast<__nv_bfloat16*>(out_hi), static_cast<__nv_bfloat16*>(out_lo), out_stride),
                       "head_norm_gated_kernel launch");
}

}  // extern "C"
