// Execution plan of the configured decoders (hybrid.h).
#pragma once

#include "dl/hybrid.h"
#include "dl/internal.h"
#include "dl/plan.h"

#include <cuda_runtime.h>

#include <memory>
#include <span>
#include <vector>

namespace dl::nn {

inline int code_of(DType dtype) { return dtype == DType::bf16 ? B200_BF16 : B200_F32; }
inline cudaStream_t cuda_stream(int device) { return static_cast<cudaStream_t>(runtime::stream(device)); }
inline float* f32(const Tensor& t) { return static_cast<float*>(t.mutable_data()); }
inline Tensor host_zeros(Shape shape, TensorOptions options) { return zeros(std::move(shape), options); }
Tensor to_f32(const Tensor& t);

// Fixed execution plan: packed weights, persistent workspaces, and per layer run
//     state space:       in-projection -> convolution + recurrence -> gated group norm -> out-projection + residual + next norm
//     latent attention:  [dq | dkv | g] projection -> norms, rotation, append -> query up-projection -> absorbed query
//                        -> attention -> value up-projection + gate -> out-projection + residual + next norm
//     feed-forward:      gate/up + SiLU * up -> down-projection + residual + next norm
//     parallel layer:    [q | k | v | g | gate/up or router, shared up] projection -> norms, rotation, append, activation, router
//                        -> attention + gate -> (experts + residual) -> [o | down] projection of both sublayers + residual + next norm
//     sandwich layer:    [q | k | v | g | right g, v, k, q] projection -> norms, rotation, append -> attention + gate
//                        -> (recurrence -> norm + gate) -> [o | right o] projection -> norm, residual, next norm
//                        -> gate/up + clamped units -> down-projection -> norm, residual, next norm
//                           or router -> experts, norm, residual, next norm
//     layer with norms behind it alone: as a sandwich layer, with the stream itself in the place of the norms before the sublayers; a delta
//                        rule in the place of the attention: [g | v | k | q | a | b] projection -> convolution + recurrence -> norm + gate
// bf16 models run the projections on the shadow protocol (activations as bf16 hi + lo planes).  The projection that finishes the
// residual stream also writes the next norm: a Dynamic Tanh norm as its result, an RMS norm as weighted rows and partial sums of
// squares, from which the consumer takes the row's factor.  f32 models and sizes the shadow kernels do not take run the same kernels
// with f32 activations and stand-alone norms.
class HybridPlan {
public:
    explicit HybridPlan(HybridDecoder& owner) : owner_(owner) {}

    void refresh();
    void reserve(Index rows, Index max_length, const HybridCache& cache, const b200_rows& pass);
    bool shadows_for(Index rows) const;
    // ids on the device; `pass` describes the rows.  Leaves the residual stream in h_ and (shadow form) its final norm in the planes.
    void run(const Index* ids, const b200_rows& pass, HybridCache& cache, Index max_length, void* stream, std::vector<float>* trail = nullptr);
    // The rows of the last run become part of the cache.
    void advance(const b200_rows& pass, HybridCache& cache, void* stream);
    // Logits of the last run's rows.
    void logits(Index rows, float* out, void* stream);
    // Logits of `count` rows of the last run, picked by device indices.
    void logits_of(const std::int32_t* index, Index count, float* out, void* stream);
    bool prepare_choice(Index rows);
    void choose(Index rows, const TokenFeedback& feedback, void* stream);
    std::uint64_t buffer_epoch() const { return epoch_; }
    void set_user(const void* user) { user_ = user; }
    const void* user() const { return user_; }
    int device() const { return owner_.embed().device().index; }
    bool norms_behind() const { return owner_.design().form == LayerForm::sandwich || owner_.design().form == LayerForm::behind; }

    // Pass descriptions: host arrays -> one device block.
    struct PassMaps {
        Tensor block;
        std::shared_ptr<runtime::Storage> staging;
        b200_rows describe(std::span<const Index> slots, std::span<const Index> counts, HybridCache& cache, int device);
    };
    PassMaps maps;

private:
    struct Norm { Tensor weight, bias; float alpha = 1.0f; bool rms = false; };
    // Rows as bf16 planes; `parts` partial sums of squares per row (in squares_) when an RMS norm's factor is still to be applied.
    struct Planes { Tensor hi, lo; Index parts = 0; };
    struct Layer {
        Norm norm1, norm2;
        const void *in, *out, *down;                // bound to the modules' tensors
        Tensor wide, gate_up, w_key;                // concatenated first projection, interleaved feed-forward, per-head transposed keys
        const void *uq, *w_value;
        Tensor conv, conv_bias, dt_bias, a_log, d, gated_norm, q_norm, kv_norm;   // f32
        Index wide_out, inner, mixed_out;           // rows of the first projection; input width of the out-projection
        // grouped-query attention
        Tensor q_bias, k_bias, sink;                // f32
        // norms behind the sublayers, router and recurrence beside the attention (sandwich layers)
        Norm after1, after2;
        Tensor router, router_bias, correction, decay, right_norm, talk;
        Index lightning_column = 0;                 // where its [g | v | k | q] start in a projected row
        b200_clamped_unit unit{};
        // parallel layers
        Tensor joint, experts_up, experts_down;     // [o | down] columns side by side; the experts' matrices one below the other
        Index attention_columns = 0;                // rows of `wide` before the feed-forward's (q | k | v | g, padded)
        Index attended = 0, units = 0;              // columns of the out-projection's input: attention, feed-forward units
        Index unit_column = 0, router_column = 0;   // where their projections start in a projected row
    };
    // What a projection that finishes the residual stream leaves for its successor: a norm's planes, the rows' own planes, or nothing.
    struct After { const Norm* norm; bool raw; };
    Norm pack_norm(const RowNorm& n, double scale = 1.0) const;
    void pack_attention(const GroupedAttentionMixer& mixer, Layer& layer) const;
    void pack_experts(const MixtureOfExperts& mixture, Layer& layer) const;
    void pack_parallel(const HybridLayer& module, Layer& layer) const;
    void pack_sandwich(const HybridLayer& module, Layer& layer) const;
    void pack_delta(const DeltaMixer& mixer, Layer& layer) const;
    // The recurrence of a delta layer from its projected rows to the input of its out-projection.
    void run_delta(std::size_t run, const b200_rows& pass, HybridCache& cache, void* stream);
    void reserve_attention(Index rows, Index max_length, const HybridCache& cache, const b200_rows& pass);
    void run_sandwich(const Index* ids, const b200_rows& pass, HybridCache& cache, Index max_length, void* stream, std::vector<float>* trail);
    // Everything of a parallel layer up to its out-projection; returns the residual that the out-projection adds to.
    const float* run_parallel(std::size_t run, const float* in, const b200_rows& pass, HybridCache& cache, Index max_length, void* stream);
    b200_chunk_args chunk_args(const Layer& layer, const HybridLayer& module, const HybridCache& cache, std::size_t run, Index stride) const;
    b200_experts expert_args(const Layer& layer, const MixtureOfExperts& mixture, Index rows) const;
    // Dense feed-forwards of parallel layers: whether their units are projected together with the attention's inputs.
    bool units_beside(const HybridLayer& module, Index rows, bool planes) const;

    void linear(const float* x, Index rows, Index in, const void* w, Index out, b200_epilogue epilogue, const float* residual, float* y, void* stream, const char* what);
    // `to` receives the planes of the result: of the `next` norm, of the result itself without one, of the gated units.
    void shadow(const Planes& x, Index rows, Index in, const void* w, Index out, b200_epilogue epilogue, const float* residual, float* y, const Norm* next,
                Planes* to, void* stream, const char* what, Index to_column = 0, Index to_stride = 0, const b200_clamped_unit* unit = nullptr);
    void planes_of(const float* x, Index rows, const Norm& norm, Planes& to, void* stream);
    b200_latent_args latent_args(const Layer& layer, const LatentAttentionMixer& mixer, const HybridCache& cache, std::size_t run) const;
    void grow(Tensor& t, Shape shape, DType dtype);
    // The rows of the stream as f32, for the trail.
    void keep_rows(Index rows, std::vector<float>& trail) const;
    void grow(Planes& p, Index rows, Index width) { grow(p.hi, {rows, width}, DType::bf16); grow(p.lo, {rows, width}, DType::bf16); }

    HybridDecoder& owner_;
    std::vector<Layer> layers_;
    Norm final_norm_;
    Tensor loop_step_, loop_x_, loop_first_;
    std::uint64_t packed_version_ = ~0ull, epoch_ = 0;
    const void* user_ = nullptr;
    Tensor first_, h_, projected_, mixed_, y_, query_, absorbed_, latent_out_, plain_, plain_inner_, scratch_;
    Tensor branch_, route_logits_;            // a sublayer's result before the norm behind it; the router's outputs
    const Index* ids_ = nullptr;              // of the last run
    Planes n_, i_, x_;                        // normed rows [rows, width]; inner rows (gated, attended, activated, query latent); the stream itself
    Tensor squares_;                          // [parts][rows]
    Tensor joined_first_, entered_;           // loop_first_ of the embedding output; the stream at the start of a pass
    Tensor chunk_query_, chunk_key_, chunk_value_, chosen_, score_, rank_, counts_, expert_act_, expert_scratch_;
    bool grouped_ = false;                    // some mixture of this row count sorts its slots: counts_ [layer runs][experts] start at zero
    Tensor picked_, best_value_, best_index_;
    Planes p_;
};

}  // namespace dl::nn
