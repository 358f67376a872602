// The two model families behind the serving engine: the LFM2 executor and the layer-stack executor.
#include "step_backend.h"

#include <cuda_runtime.h>
#include <string.h>

#include <algorithm>
#include <vector>

#include "kernels.h"

namespace lfm25 {

namespace {

#define BACKEND_TRY(expression)            \
    do {                                   \
        const int32_t rc_ = (expression);  \
        if (rc_ != LFM25_OK) return rc_;   \
    } while (0)

int32_t cuda_result(cudaError_t status) {
    return status == cudaSuccess ? LFM25_OK : report_error(LFM25_ERR_CUDA, cudaGetErrorString(status));
}

class Lfm2Backend final : public StepBackend {
  public:
    Lfm2Backend(lfm25_blaslt* blaslt, const lfm25_model* model, uint32_t use_fp8, size_t state_rows)
        : blaslt_(blaslt), model_(model), use_fp8_(use_fp8), state_rows_(state_rows) {
        for (uint32_t layer = 0; layer < model->num_layers; ++layer) {
            if (!model->layers[layer].is_attention) conv_layers_.push_back(layer);
        }
    }
    ~Lfm2Backend() override { lfm25_decode_executor_destroy(executor_); }

    size_t num_pages() const override { return model_->num_pages; }
    size_t num_request_slots() const override { return model_->num_request_slots; }
    size_t vocab() const override { return kVocab; }
    size_t maximum_rows() const override { return maximum_rows_; }
    bool any_output_rows() const override { return false; }

    int32_t create_executor(size_t maximum_tokens, size_t maximum_segments) override {
        maximum_rows_ = maximum_segments;
        return lfm25_decode_executor_create_ragged(blaslt_, maximum_tokens, maximum_segments, &executor_);
    }
    int32_t create_checkpoints(size_t capacity, lfm25_conv_checkpoints** out) override {
        if (conv_layers_.empty()) return LFM25_OK;
        return lfm25_conv_checkpoints_create(conv_layers_.size(), capacity, kHidden, 2, out);
    }
    int32_t capture_state(lfm25_conv_checkpoints* pool, uint32_t checkpoint, size_t slot) override {
        for (size_t index = 0; index < conv_layers_.size(); ++index) {
            BACKEND_TRY(lfm25_conv_checkpoints_capture_layer(pool, stream(), checkpoint, index, conv_state(index), slot,
                                                             state_rows_));
        }
        return LFM25_OK;
    }
    int32_t restore_state(lfm25_conv_checkpoints* pool, uint32_t checkpoint, size_t slot) override {
        for (size_t index = 0; index < conv_layers_.size(); ++index) {
            BACKEND_TRY(lfm25_conv_checkpoints_restore_layer(pool, stream(), checkpoint, index, conv_state(index), slot,
                                                             state_rows_));
        }
        return LFM25_OK;
    }
    int32_t clear_state(size_t slot) override {
        for (size_t index = 0; index < conv_layers_.size(); ++index) {
            char* state = static_cast<char*>(conv_state(index)) + slot * kHidden * 2 * 2;
            BACKEND_TRY(cuda_result(cudaMemsetAsync(state, 0, kHidden * 2 * 2, stream())));
        }
        return LFM25_OK;
    }
    int32_t decode(const lfm25_decode_batch& batch, bool graph) override {
        // the metadata was uploaded by the caller, so the step does not advance it on the device
        return graph ? lfm25_decode_executor_step_graph(executor_, model_, &batch, use_fp8_, 0)
                     : lfm25_decode_executor_forward(executor_, model_, &batch, use_fp8_, 0);
    }
    int32_t mixed(const lfm25_ragged_batch& batch, size_t) override {
        return lfm25_decode_executor_forward_ragged(executor_, model_, &batch, use_fp8_);
    }
    int32_t download_sampled(uint32_t* host, size_t count) override {
        return lfm25_decode_executor_download_sampled(executor_, host, count);
    }
    int32_t read_logits(float* host, size_t rows) override {
        std::vector<uint16_t> bits(rows * kVocab);
        BACKEND_TRY(lfm25_decode_executor_download_logits(executor_, bits.data(), rows));
        BACKEND_TRY(cuda_result(cudaStreamSynchronize(stream())));
        for (size_t index = 0; index < bits.size(); ++index) {
            const uint32_t word = static_cast<uint32_t>(bits[index]) << 16;
            memcpy(host + index, &word, 4);
        }
        return LFM25_OK;
    }

  private:
    static constexpr size_t kHidden = 2048;
    static constexpr size_t kVocab = 65536;
    cudaStream_t stream() const { return static_cast<cudaStream_t>(lfm25_blaslt_stream(blaslt_)); }
    void* conv_state(size_t index) const { return model_->layers[conv_layers_[index]].conv_state; }

    lfm25_blaslt* blaslt_;
    const lfm25_model* model_;
    uint32_t use_fp8_;
    size_t state_rows_;
    size_t maximum_rows_ = 0;
    std::vector<uint32_t> conv_layers_;   // indices of the gated-convolution layers in the model
    lfm25_decode_executor* executor_ = nullptr;
};

class StackBackend final : public StepBackend {
  public:
    StackBackend(lfm25_blaslt* blaslt, const lfm25_stack_model* model) : blaslt_(blaslt), model_(model) {}
    ~StackBackend() override { lfm25_stack_executor_destroy(executor_); }

    size_t num_pages() const override { return model_->num_pages; }
    size_t num_request_slots() const override { return model_->num_request_slots; }
    size_t vocab() const override { return model_->vocab; }
    size_t maximum_rows() const override { return maximum_rows_; }
    bool any_output_rows() const override { return true; }

    int32_t create_executor(size_t maximum_tokens, size_t maximum_segments) override {
        maximum_rows_ = std::min(std::max<size_t>(maximum_segments, 256), maximum_tokens);
        return lfm25_stack_executor_create(blaslt_, model_, maximum_tokens, maximum_rows_, &executor_);
    }
    // One checkpoint is the slot's whole record; the pool counts in pairs of 16-bit elements.
    int32_t create_checkpoints(size_t capacity, lfm25_conv_checkpoints** out) override {
        return lfm25_conv_checkpoints_create(1, capacity, model_->record_bytes / 4, 2, out);
    }
    int32_t capture_state(lfm25_conv_checkpoints* pool, uint32_t checkpoint, size_t slot) override {
        return lfm25_conv_checkpoints_capture_layer(pool, stream(), checkpoint, 0, model_->records, slot,
                                                    model_->num_request_slots);
    }
    int32_t restore_state(lfm25_conv_checkpoints* pool, uint32_t checkpoint, size_t slot) override {
        return lfm25_conv_checkpoints_restore_layer(pool, stream(), checkpoint, 0, model_->records, slot,
                                                    model_->num_request_slots);
    }
    int32_t clear_state(size_t slot) override {
        char* record = static_cast<char*>(model_->records) + slot * model_->record_bytes;
        return cuda_result(cudaMemsetAsync(record, 0, model_->record_bytes, stream()));
    }
    int32_t decode(const lfm25_decode_batch& batch, bool graph) override {
        return graph ? lfm25_stack_executor_step_graph(executor_, &batch, 0)
                     : lfm25_stack_executor_forward(executor_, &batch, 0);
    }
    int32_t mixed(const lfm25_ragged_batch& batch, size_t num_output_rows) override {
        return lfm25_stack_executor_forward_ragged(executor_, &batch, num_output_rows);
    }
    int32_t download_sampled(uint32_t* host, size_t count) override {
        return lfm25_stack_executor_download_sampled(executor_, host, count);
    }
    int32_t read_logits(float* host, size_t rows) override {
        return lfm25_stack_executor_read_logits(executor_, host, rows);
    }

  private:
    cudaStream_t stream() const { return static_cast<cudaStream_t>(lfm25_blaslt_stream(blaslt_)); }

    lfm25_blaslt* blaslt_;
    const lfm25_stack_model* model_;
    size_t maximum_rows_ = 0;
    lfm25_stack_executor* executor_ = nullptr;
};

}  // namespace

std::unique_ptr<StepBackend> lfm2_backend(lfm25_blaslt* blaslt, const lfm25_model* model, uint32_t use_fp8,
                                          size_t state_rows) {
    return std::make_unique<Lfm2Backend>(blaslt, model, use_fp8, state_rows);
}

std::unique_ptr<StepBackend> stack_backend(lfm25_blaslt* blaslt, const lfm25_stack_model* model) {
    return std::make_unique<StackBackend>(blaslt, model);
}

}  // namespace lfm25
