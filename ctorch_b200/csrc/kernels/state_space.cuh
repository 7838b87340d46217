// What the recurrences with a state per head share (state_space.cu: Mamba-2 and lightning attention; delta_rule.cu: the gated delta rule):
// the layer's view, decays, the convolution of a step, staging and packed arithmetic.
#pragma once

#include "mma.cuh"
#include "rows.cuh"

namespace b200 {

struct SsmParams {
    int heads, vdim, state, groups, taps, channels, stride;
    const float *conv_weight, *conv_bias, *dt_bias, *a_log, *d;
    float *conv_state, *ssm_state;
    const float* projected;
    float *mixed, *y;
    const float* fixed_decay;   // [heads] or NULL: step sizes and decays come from the projection
};

__device__ __forceinline__ float softplus(float v) { return v > 20.0f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float sigmoid_exact(float v) { return 1.0f / (1.0f + expf(-v)); }

// Input of the convolution at `position` of a slot, from the ring of earlier passes (zero before the sequence's start).
__device__ __forceinline__ float ring_input(const SsmParams& p, int slot, int position, int channel) {
    if (position < 0) return 0.0f;
    return p.conv_state[(static_cast<int64_t>(slot) * p.taps + position % p.taps) * p.channels + channel];
}

// Step size and decay of a head for one projected row.
struct StepRate { float dt, decay; };
__device__ __forceinline__ StepRate step_rate(const SsmParams& p, const float* row, int head) {
    if (p.fixed_decay) return {1.0f, __ldg(p.fixed_decay + head)};
    const float dt = softplus(row[p.heads * p.vdim + p.channels + head] + p.dt_bias[head]);
    return {dt, expf(-expf(p.a_log[head]) * dt)};
}

constexpr int kStepThreads = 256;

// Convolved channels of one head for one token: [x: vdim | B: state | C: state] into `mixed`, and the token's inputs into the
// slot's ring (B and C are shared by the heads of a group: its first head writes them).
__device__ __forceinline__ void convolve_head(const SsmParams& p, const float* in, int slot, int position, int head, float* mixed) {
    const int P = p.vdim, N = p.state, inner = p.heads * P, per_group = p.heads / p.groups, group = head / per_group;
    const bool shared_writer = head == group * per_group;
    // the ring entry of the current token; entry of the token `back` places before: ring_at - back, wrapped
    const int ring_at = position % p.taps;
    float* const ring = p.conv_state + static_cast<int64_t>(slot) * p.taps * p.channels;
    for (int i = threadIdx.x; i < P + 2 * N; i += kStepThreads) {
        const int c = i < P ? head * P + i : i < P + N ? inner + group * N + (i - P) : inner + (p.groups + group) * N + (i - P - N);
        const float now = in[inner + c];
        if (!p.conv_weight) {
            mixed[i] = now * sigmoid_exact(now);
            continue;
        }
        const float* weight = p.conv_weight + c * p.taps;
        float acc = p.conv_bias[c];
#pragma unroll 4
        for (int j = 0; j < p.taps - 1; ++j) {
            const int back = p.taps - 1 - j, at = ring_at < back ? ring_at - back + p.taps : ring_at - back;
            const float old = position < back ? 0.0f : ring[at * p.channels + c];
            acc = fmaf(weight[j], old, acc);
        }
        acc = fmaf(weight[p.taps - 1], now, acc);
        mixed[i] = acc * sigmoid_exact(acc);
        if (i < P || shared_writer) ring[ring_at * p.channels + c] = now;
    }
}

__device__ __forceinline__ void bulk_store(void* dst, const void* src, uint32_t bytes) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(smem_u32(src)), "r"(bytes) : "memory");
    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

// Packed f32 pairs: two independent IEEE operations per instruction.
__device__ __forceinline__ uint64_t pack2(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ void copy_async_4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// The gated delta rule over convolved channels (in p.mixed, except steps that convolve themselves); see delta_rule.cu.
int launch_delta_step(const SsmParams& p, const RowsView& rows, cudaStream_t stream);
bool delta_step_streams(const SsmParams& p, const RowsView& rows, int sms);
int launch_delta_step_stream(const SsmParams& p, const RowsView& rows, int sms, int32_t* status, cudaStream_t stream);
int launch_delta_scan(const SsmParams& p, const RowsView& rows, cudaStream_t stream);

}  // namespace b200
