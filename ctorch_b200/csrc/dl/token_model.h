// What the generation loop needs of a model: token ids in, logits or chosen ids out, with a cache behind it that the model owns or
// borrows.  Implemented by the grouped-query decoder with its embedding and output layers (DecoderTokenModel, plan.cpp) and by the
// hybrid decoder (HybridTokenModel, hybrid.cpp).
#pragma once

#include "dl/dl.h"

#include <cstdint>

namespace dl::nn {

// Where the token loop keeps its state on the device (see b200_token_feedback).
struct TokenFeedback {
    Index* next;
    Index* ids;
    Index* history;
    Index history_rows;
    std::int32_t* counter;
};

class TokenModel {
public:
    virtual ~TokenModel() = default;
    virtual int device() const = 0;
    virtual Index vocabulary() const = 0;               // token ids the embedding holds
    virtual Index outputs() const = 0;                  // logits per position
    virtual std::uint64_t version() const = 0;          // moves with the parameters
    virtual void refresh() = 0;                         // packs weights again when they moved
    // Throws unless every sequence of the batch has room for `length` more tokens.
    virtual void validate(Index batch, Index length) = 0;
    virtual std::uint64_t buffer_epoch() const = 0;     // moves when a workspace of the step was reallocated
    // Prompt ids [batch, P] on the device into the cache, sequence s with its first lengths[s] tokens (all P without lengths);
    // the logits of every sequence's last token to `logits` [batch, outputs].  Returns with the work complete.
    virtual void prefill(const Tensor& prompt, std::span<const Index> lengths, float* logits) = 0;
    // Workspaces of a single-token step, before it is enqueued or captured; whether choose() serves it.
    virtual bool prepare_step(Index batch) = 0;
    // Enqueue one token of every sequence: embedding and layers.  The cache lengths move on with advance() or choose().
    virtual void step(const Index* ids, Index batch, void* stream) = 0;
    virtual void advance(Index batch, void* stream) = 0;
    virtual void logits(Index batch, float* out, void* stream) = 0;                              // of the last step
    virtual void choose(Index batch, const TokenFeedback& feedback, void* stream) = 0;           // logits + greedy choice + advance
    virtual void commit(Index steps) = 0;               // host mirror of the lengths after `steps` enqueued steps
    // Who ran the model last: the final hidden state in the workspaces belongs to that user.
    virtual void set_user(const void* user) = 0;
    virtual const void* user() const = 0;
};

// Optional per-launch event trail (Generation::profile_step); kinds: 0 linear, 1 attention, 2 other.
void probe(int kind);

}  // namespace dl::nn
