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

// With N(x; w) = x / sqrt(mean(x^2) + eps) * (shift + w), per row:
//   x = residual (or the embedding row of token_ids), plus N(update; post_norm) when there is an update
//   residual_out = x,  out = N(x; norm)            -- either may be left out
// Row i reads row rows[i] (rows == nullptr: i) of residual and update; residual_out may be the buffer of residual.
struct ResidualPostNormLaunch {
    Activation type;
    const float* residual;         // [T, width]; unused with an embedding
    const void* update;            // [T, width] activations, or nullptr
    const void* post_norm;         // bf16 [width]
    const uint32_t* token_ids;     // [T] with `embedding`, else nullptr
    const void* embedding;         // bf16 [vocab, width] or nullptr
    size_t vocab;
    const void* norm;              // bf16 [width]
    const uint32_t* rows;
    float* residual_out;           // [num_rows, width] or nullptr
    void* out;                     // [num_rows, width] activations or nullptr
    size_t num_rows;
    size_t num_tokens;
    size_t width;
    float shift;
    float eps;
};
cudaError_t launch_residual_post_norm(cudaStream_t stream, const ResidualPostNormLaunch& launch);

// z <- relu(z)^2 in place
cudaError_t launch_squared_relu(cudaStream_t stream, Activation type, void* z, size_t count);

// out[t, c] = a N(z)[c] + b N(z^2)[c] + c N(z^3)[c] + e with N the unweighted RMS norm of the row; columns
// width .. width + pad - 1 of `out` are set to zero.
cudaError_t launch_poly_norm(cudaStream_t stream, Activation type, const void* z, size_t z_pitch, void* out,
                             size_t out_pitch, size_t rows, size_t width, size_t pad, const float coefficients[4],
                             float eps);

// Greedy choice: index of the row's largest logit, the lowest index among equals; NaN never wins.  A cap on the logits
// keeps their order, so the choice is made before it.
cudaError_t launch_argmax_rows(cudaStream_t stream, Activation type, const void* logits, size_t pitch,
                               uint32_t* sampled, size_t rows, size_t vocab);

// out[r, v] = the logit as f32; softcap > 0: softcap * tanh(logit / softcap)
cudaError_t launch_export_logits(cudaStream_t stream, Activation type, const void* logits, size_t pitch, float* out,
                                 size_t rows, size_t vocab, float softcap);

// y[m, n] = sum_k x[m, k] w[n, k] with plain 32-bit multiply-adds: the matrix product of the f32 activation type and
// of bf16 shapes that the tensor-core paths cannot take.
cudaError_t launch_linear_simt(cudaStream_t stream, Activation type, const void* x, const void* weight, void* y,
                               size_t m, size_t n, size_t k);

// One matrix product per head: y[t, h, n] = sum_k x[t, h, k] w[h, n, k] (gate: times sigmoid(gate[t, h * n_size + n])).
struct HeadLinearLaunch {
    Activation type;
    const void* x;                 // activations: token t, head h at x + t * x_pitch + h * x_head
    size_t x_pitch, x_head;
    const void* weight;            // bf16: head h, output n, input k at weight + h * w_head + n * w_n + k * w_k
    size_t w_head, w_n, w_k;       // w_n or w_k is 1
    void* y;                       // activations: y + t * y_pitch + h * n
    size_t y_pitch;
    const void* gate;              // activations, token t at gate + t * gate_pitch, or nullptr
    size_t gate_pitch;
    size_t tokens, n, k;
    uint32_t heads;
};
cudaError_t launch_head_linear(cudaStream_t stream, const HeadLinearLaunch& launch);

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

// -------------------------------------------------------------------------------------------- latent attention

struct LatentAttentionShape {
    uint32_t heads, dim, rot_dim, vdim, kv_rank;
    float scale;
};

// The projections of latent attention: out = N(query latent) * query_norm; N(latent) * latent_norm and the rotated key
// part into the paged cache.  `projected` rows hold query latent | latent | key part, the latter two from `latent_column`.
struct LatentProjectionLaunch {
    Activation type;
    const void* projected;
    size_t pitch;
    uint32_t q_rank, kv_rank, rot_dim, rot_dims;
    size_t latent_column;
    bool append;                   // false: the cache is another layer's, only the query latent is wanted
    const void* query_norm;        // bf16 [q_rank]
    const void* latent_norm;       // bf16 [kv_rank]
    const float* inv_freq;         // f32 [rot_dims / 2]
    const uint32_t* positions;
    const int64_t* physical_slots; // negative = do not append
    void* query_out;               // [T, q_rank]
    void* latent_cache;            // [pages, 16, kv_rank]
    void* key_cache;               // [pages, 16, rot_dim]
    size_t num_tokens;
    size_t num_pages;
    float eps;
};
cudaError_t launch_latent_projection(cudaStream_t stream, const LatentProjectionLaunch& launch);

// Rotates entries 0 .. rot_dims - 1 behind the first `dim` of every head, in place; query [T, heads, dim + rot_dim] in rows
// `pitch` apart.
cudaError_t launch_rotate_queries(cudaStream_t stream, Activation type, void* query, size_t pitch, const float* inv_freq,
                                  const uint32_t* positions, size_t tokens, uint32_t heads, uint32_t dim,
                                  uint32_t rot_dim, uint32_t rot_dims);

// Attention against the latents themselves: the key up-projection has been moved to the query side, so one latent vector
// and one rotated key per token serve all heads, and the output is the weighted latent of every head.
struct LatentAttentionLaunch {
    Activation type;
    LatentAttentionShape shape;
    const void* absorbed;          // [T, heads, kv_rank]
    const void* query;             // [T, heads, dim + rot_dim], rows query_pitch apart: the last rot_dim, rotated
    size_t query_pitch;
    const void* latent_cache;
    const void* key_cache;
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* request_slots; // [T]
    const uint32_t* positions;     // [T]
    const uint32_t* token_order;   // a permutation of the tokens, in which they are started, or nullptr
    size_t tokens;
    size_t context;                // longest context among them when known, else 0
    unsigned int* status;
    void* out;                     // [T, heads, kv_rank]
};
cudaError_t launch_latent_attention(cudaStream_t stream, const LatentAttentionLaunch& launch);

// Row of a step's context scratch at which each segment's keys start: segment s takes ceil(context / 64) * 64 rows in
// order; the segments from `first_segment` on.  bases has num_segments + 1 entries.
cudaError_t launch_context_bases(cudaStream_t stream, const StackSegments& segments, const uint32_t* positions,
                                 size_t first_segment, uint32_t* bases);

// Copies the cached latents and rotated keys of those segments' contexts into contiguous rows; rows behind a context are
// cleared.
struct GatherContextLaunch {
    Activation type;
    StackSegments segments;
    size_t first_segment;
    const uint32_t* bases;
    const uint32_t* positions;
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    uint32_t kv_rank, rot_dim;
    const void* latent_cache;
    const void* key_cache;
    void* latents;                 // [rows, kv_rank]
    void* keys;                    // [rows, rot_dim]
    size_t rows;
};
cudaError_t launch_gather_context(cudaStream_t stream, const GatherContextLaunch& launch);

// Prompt attention over keys and values that were formed from the gathered latents: `expanded` rows hold heads * dim key
// columns, then heads * vdim value columns.
struct ExpandedAttentionLaunch {
    Activation type;
    LatentAttentionShape shape;
    const void* query;             // [T, heads, dim + rot_dim], rows query_pitch apart
    size_t query_pitch;
    const void* expanded;
    size_t expanded_pitch;
    const void* keys;              // [rows, rot_dim]
    const uint32_t* bases;
    size_t rows;
    size_t first_segment;
    StackSegments segments;
    const uint32_t* positions;
    const void* gate;              // activations, token t at gate + t * gate_pitch, heads * vdim columns
    size_t gate_pitch;
    unsigned int* status;
    void* out;                     // activations, rows out_pitch apart, heads * vdim columns
    size_t out_pitch;
};
bool expanded_attention_supports(Activation type, const LatentAttentionShape& shape, size_t out_pitch, size_t gate_pitch,
                                 size_t expanded_pitch);
cudaError_t launch_expanded_attention(cudaStream_t stream, const ExpandedAttentionLaunch& launch);

// ---------------------------------------------------------------------------------------------- state-space mixer

// out[t, c] = silu(sum_j conv[j, c] x[t - taps + 1 + j, c] + bias[c]) over `channels` columns of x; the last taps - 1
// inputs live in `record` as [taps - 1, channels] activations, oldest first.
struct ChannelConvLaunch {
    Activation type;
    StackSegments segments;
    const void* x;
    size_t pitch;
    const void* conv;              // bf16 [taps, channels]
    const void* bias;              // bf16 [channels]
    uint32_t taps;
    StackRecord record;
    void* out;                     // [T, channels]
    size_t channels;
};
cudaError_t launch_channel_conv(cudaStream_t stream, const ChannelConvLaunch& launch);

// Per head S <- exp(-exp(log_rate) dt) S + dt B x^T, y = S^T C + skip x with dt = softplus(raw + step_bias); `mixed` rows
// hold x [heads, vdim] | B [groups, size] | C [groups, size].  State: f32 [heads, size, vdim] in `record`.
struct StateSpaceLaunch {
    Activation type;
    StackSegments segments;
    size_t decode_tokens;          // the first decode_tokens segments hold one token each
    uint32_t heads, groups, size, vdim;
    const void* mixed;
    size_t mixed_pitch;
    const void* raw_step;          // activations: token t at raw_step + t * step_pitch, heads columns
    size_t step_pitch;
    const void* step_bias;         // bf16 [heads]
    const void* log_rate;
    const void* skip;
    StackRecord record;
    void* out;                     // [T, heads * vdim]
};
constexpr uint32_t kStateSpaceMaxSize = 512;
cudaError_t launch_state_space(cudaStream_t stream, const StateSpaceLaunch& launch);

// out = N(y silu(z)) * norm, N over each of `groups` equal parts of the row on its own.
struct GatedGroupNormLaunch {
    Activation type;
    const void* y;                 // [T, width]
    const void* z;                 // activations, rows z_pitch apart
    size_t z_pitch;
    const void* norm;              // bf16 [width]
    void* out;                     // activations, rows out_pitch apart
    size_t out_pitch;
    size_t tokens, width;
    uint32_t groups;
    float eps;
};
cudaError_t launch_gated_group_norm(cudaStream_t stream, const GatedGroupNormLaunch& launch);

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
