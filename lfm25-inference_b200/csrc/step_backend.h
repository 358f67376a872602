// What the serving engine needs of a model family: steps, the recurrent state of a request slot, and its checkpoints.
// The engine owns everything else (slots, pages, prefix index, planning, token bookkeeping).
#pragma once

#include <stddef.h>
#include <stdint.h>

#include <memory>

#include "../../include/lfm25_b200.h"

namespace lfm25 {

class StepBackend {
  public:
    virtual ~StepBackend() = default;
    virtual size_t num_pages() const = 0;
    virtual size_t num_request_slots() const = 0;
    virtual size_t vocab() const = 0;
    // rows that may get logits in one step, and whether they may be any tokens (else: each segment's last one)
    virtual size_t maximum_rows() const = 0;
    virtual bool any_output_rows() const = 0;
    virtual int32_t create_executor(size_t maximum_tokens, size_t maximum_segments) = 0;
    // a pool that holds the recurrent state of `capacity` prefixes; *out stays null when there is no such state
    virtual int32_t create_checkpoints(size_t capacity, lfm25_conv_checkpoints** out) = 0;
    virtual int32_t capture_state(lfm25_conv_checkpoints* pool, uint32_t checkpoint, size_t slot) = 0;
    virtual int32_t restore_state(lfm25_conv_checkpoints* pool, uint32_t checkpoint, size_t slot) = 0;
    virtual int32_t clear_state(size_t slot) = 0;
    virtual int32_t decode(const lfm25_decode_batch& batch, bool graph) = 0;
    virtual int32_t mixed(const lfm25_ragged_batch& batch, size_t num_output_rows) = 0;
    virtual int32_t download_sampled(uint32_t* host, size_t count) = 0;
    virtual int32_t read_logits(float* host, size_t rows) = 0;   // f32 [rows, vocab], synchronises
};

std::unique_ptr<StepBackend> lfm2_backend(lfm25_blaslt* blaslt, const lfm25_model* model, uint32_t use_fp8,
                                          size_t state_rows);
std::unique_ptr<StepBackend> stack_backend(lfm25_blaslt* blaslt, const lfm25_stack_model* model);

}  // namespace lfm25
