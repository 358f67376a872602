// Host-side launch functions of the layer-stack kernels: the mechanisms that a model described layer by layer
// (lfm25_stack_model) is assembled from.  Internal to the library; arguments are validated by the executor.
//
// Every kernel exists for two activation types: bf16 (serving) and f32 (everything in 32 bits).  Weights are bf16 in
// both; norms, softmax, rotation, the residual stream and recurrent state are always 32-bit.
#pragma once

#include <cuda_runtime.h>
#include <stddef.h>
#include <stdint.h>

namespace lfm25 {

enum class Activation : uint32_t { kBf16 = 0, kF32 = 1 };
inline size_t activation_bytes(Activation type) { return type == Activation::kF32 ? 4 : 2; }

// Which tokens of a step belong together.  `offsets` == nullptr: every token is a segment of its own and `slots` is
// indexed by token (a decode step); otherwise segment s holds tokens offsets[s] .. offsets[s + 1] - 1.
struct StackSegments {
    const uint32_t* offsets;
    const uint32_t* slots;       // request slot per segment
    size_t num_segments;
    size_t num_tokens;
    size_t num_request_slots;
};

// The recurrent state of all layers, one record of `stride` bytes per request slot; a layer's part starts `offset`
// bytes into the record.
struct StackRecord {
    void* base;
    size_t stride;
    size_t offset;
};

// x = residual + update (or the embedding row of token_ids), h = norm(x) * mixer_norm, n = norm(x) * ff_norm,
// mixed = h + causal convolution of h over the sequence.  The convolution's last taps - 1 inputs live in `record` as
// [taps - 1, width] activations, oldest first.
struct ResidualNormConvLaunch {
    Activation type;
    StackSegments segments;
    const float* residual;         // [T, width]; unused with an embedding
    const void* update;            // [T, width] activations, may be nullptr
    const uint32_t* token_ids;     // [T] with `embedding`, else nullptr
    const void* embedding;         // bf16 [vocab, width] or nullptr
    size_t vocab;
    const void* mixer_norm;        // bf16 [width]
    const void* ff_norm;           // bf16 [width], nullptr = no feed-forward input wanted
    const void* conv;              // bf16 [taps, width], tap-major, the last row weighs the current token
    uint32_t taps;
    StackRecord record;
    float* residual_out;           // [T, width], not the same buffer as `residual`
    void* mixed_out;               // [T, width]
    void* ff_out;                  // [T, width]
    size_t width;
    float eps;
};
cudaError_t launch_residual_norm_conv(cudaStream_t stream, const ResidualNormConvLaunch& launch);

// out[i] = norm(residual[r] + update[r]) * weight with r = rows[i] (rows == nullptr: r = i)
cudaError_t launch_residual_norm_rows(cudaStream_t stream, Activation type, const float* residual, const void* update,
                                      const void* weight, const uint32_t* rows, void* out, size_t num_rows,
                                      size_t num_tokens, size_t width, float eps);

// out[t, c] = a N(z)[c] + b N(z^2)[c] + c N(z^3)[c] + e with N the unweighted RMS norm of the row; columns
// width .. width + pad - 1 of `out` are set to zero.
cudaError_t launch_poly_norm(cudaStream_t stream, Activation type, const void* z, size_t z_pitch, void* out,
                             size_t out_pitch, size_t rows, size_t width, size_t pad, const float coefficients[4],
                             float eps);

// Greedy choice: index of the row's largest logit, the lowest index among equals; NaN never wins.
cudaError_t launch_argmax_rows(cudaStream_t stream, Activation type, const void* logits, size_t pitch,
                               uint32_t* sampled, size_t rows, size_t vocab);

// y[m, n] = sum_k x[m, k] w[n, k] with plain 32-bit multiply-adds: the matrix product of the f32 activation type and
// of bf16 shapes that the tensor-core paths cannot take.
cudaError_t launch_linear_simt(cudaStream_t stream, Activation type, const void* x, const void* weight, void* y,
                               size_t m, size_t n, size_t k);

// ---------------------------------------------------------------------------------------------------- attention

struct StackAttentionShape {
    uint32_t heads, kv_heads, dim, vdim;
    uint32_t rot_dims;   // leading dimensions of each head that are rotated, 0 = none
    uint32_t chunk;      // position i sees j <= i with i / chunk == j / chunk; 0 = every j <= i
    float scale;
};

// Biases, RMS norm over the whole query (key) projection, rotary positions, append to the paged cache.
// `projected` rows hold q | k | v; key cache [pages, kv_heads, 16, dim], value cache [pages, kv_heads, 16, vdim].
struct ProjectionNormRopeLaunch {
    Activation type;
    StackAttentionShape shape;
    const void* projected;
    size_t pitch;
    const void* bias;              // bf16, q | k | v, or nullptr
    const void* query_norm;        // bf16 [heads * dim]
    const void* key_norm;          // bf16 [kv_heads * dim]
    const float* inv_freq;         // f32 [rot_dims / 2]
    const uint32_t* positions;
    const int64_t* physical_slots; // negative = do not append
    void* query_out;               // [T, heads * dim]
    void* key_cache;
    void* value_cache;
    size_t num_tokens;
    size_t num_pages;
    float eps;
};
cudaError_t launch_projection_norm_rope(cudaStream_t stream, const ProjectionNormRopeLaunch& launch);

struct StackAttentionLaunch {
    Activation type;
    StackAttentionShape shape;
    const void* query;             // [T, heads * dim]
    const void* key_cache;
    const void* value_cache;
    const uint32_t* block_tables;  // [rows, stride]
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* request_slots; // [T]
    const uint32_t* positions;     // [T]
    StackSegments segments;
    // The first decode_tokens tokens are segments of one token; decode_context is the longest context among them (what
    // their key range is split by).
    size_t decode_tokens;
    size_t decode_context;
    unsigned int* status;          // device status words of the bounded waits
    void* out;                     // activations, rows out_pitch apart, heads * vdim columns
    size_t out_pitch;
};
cudaError_t launch_stack_attention(cudaStream_t stream, const StackAttentionLaunch& launch);

// ---------------------------------------------------------------------------------------------------- delta rule

// The generalised delta rule over whole segments: decay, removal rate and unit key from the projections, the
// recurrence, the per-head norm and the output gate.  `projected` rows hold r | k | v | g | a | z (heads * dim columns
// each, z: rank).  State: f32 [heads, value dim, key dim] in `record`.
struct DeltaRuleLaunch {
    Activation type;
    StackSegments segments;
    size_t decode_tokens;          // the first decode_tokens segments hold one token each
    uint32_t heads, dim, rank;
    const void* projected;
    size_t pitch;
    const void* decay_up;          // bf16 [heads * dim, rank]
    const void* decay_base;        // bf16 [heads * dim]
    const void* removal_bias;      // bf16 [heads * dim]
    const void* norm;              // bf16 [heads * dim]
    StackRecord record;
    float* raw;                    // f32 [T, heads * dim] scratch, needed when delta_rule_needs_scratch(dim)
    void* out;                     // activations, rows out_pitch apart, heads * dim columns
    size_t out_pitch;
    float eps;
};
constexpr uint32_t kDeltaMaxDim = 256;
bool delta_rule_needs_scratch(uint32_t dim);
cudaError_t launch_delta_rule(cudaStream_t stream, const DeltaRuleLaunch& launch);

}  // namespace lfm25
