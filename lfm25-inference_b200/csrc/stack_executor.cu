// Steps of a layer-stack model: the launches of one decode or mixed step on fixed-address scratch, and decode steps
// replayed from CUDA graphs.
//
// Parallel arrangement, per layer:
//             residual sum + both norms + input convolution  ->  mixer projections (one GEMM)  ->  mixer
//             feed-forward up projection  ->  activation                                        \ side by side in one
//             [mixer output | activation] x [W_o | W_down]^T (one GEMM, f32 accumulation)       / buffer
// The residual stream stays in f32 and ping-pongs between two buffers, because a tile of the first kernel also reads
// rows of its neighbours.
// Sandwich arrangement, per sublayer:
//             residual sum with the normed output of the sublayer before + norm (one kernel)  ->  mixer or feed-forward
#include <stdio.h>

#include <algorithm>
#include <new>
#include <vector>

#include "../../include/lfm25_b200.h"
#include "blaslt_handle.h"
#include "kernels.h"
#include "options.h"
#include "stack_kernels.h"
#include "step_graphs.h"

using lfm25::Activation;

struct lfm25_stack_executor {
    lfm25_blaslt* blaslt;
    const lfm25_stack_model* model;
    Activation type;
    size_t maximum_tokens;
    size_t maximum_rows;
    uint32_t depth;            // layers that run, num_layers unless a test asked for fewer
    void* allocation;
    float* residual[2];        // [T, width]
    void* mixed;               // [T, width]: mixer input
    void* normalized;          // [T, width]: feed-forward input
    void* projected;           // [T, widest projection]
    void* query;               // [T, widest heads * dim]
    void* up;                  // [T, widest ff]
    void* joined;              // [T, widest output.k]: mixer output | activation
    void* update;              // [T, width]
    void* head_input;          // [R, width]
    void* logits;              // [R, head.n], before a cap
    float* raw;                // [T, widest heads * dim] when a delta rule needs it
    void* compressed;          // [T, widest q_rank]: latent attention's query latent
    void* absorbed;            // [T, widest heads * kv_rank]: queries against latents
    void* weighted;            // [T, widest heads * kv_rank]: weighted latents
    void* context_latents;     // [C, widest kv_rank]: contiguous contexts of a step's prompts
    void* context_keys;        // [C, widest rot_dim]
    void* expanded;            // [C, widest latent_up.n]: their keys and values
    uint32_t* context_bases;   // [T + 1]
    uint32_t* token_order;     // [T]: the tokens that attend to latents, longest context first
    void* convolved;           // [T, widest channels] of a state-space mixer
    void* scanned;             // [T, widest heads * vdim]
    size_t context_capacity = 0;
    const void* last_post = nullptr;   // norm between `update` and the residual stream of the last step
    uint32_t* sampled;         // [R]
    float* exported = nullptr; // [rows, vocab] logits on their way to the host, grown when asked for
    size_t exported_bytes = 0;
    size_t last_tokens = 0;
    const float* last_residual = nullptr;
    std::vector<unsigned char> staging;
    lfm25::StepGraphs graphs;
};

namespace {

int32_t cuda_failure(cudaError_t status, const char* what) {
    char message[200];
    snprintf(message, sizeof message, "%s: %s", what, cudaGetErrorString(status));
    return lfm25::report_error(LFM25_ERR_CUDA, message);
}

#define STACK_TRY(expression)              \
    do {                                   \
        const int32_t rc_ = (expression);  \
        if (rc_ != LFM25_OK) return rc_;   \
    } while (0)
#define STACK_CUDA(expression, what)                                \
    do {                                                            \
        const cudaError_t status_ = (expression);                   \
        if (status_ != cudaSuccess) return cuda_failure(status_, what); \
    } while (0)

// Rows of context scratch: enough for the contexts of a few full steps, bounded in bytes.  Prompts whose contexts do not
// fit attend to the cached latents directly.
constexpr size_t kContextBytes = size_t(1) << 30;
// Portions of at most this many tokens per prompt (on average) are cheaper against the latents than against keys and
// values formed from them.
constexpr size_t kShortPortion = 4;

size_t mixer_columns(const lfm25_stack_layer& layer) {
    return static_cast<size_t>(layer.heads) * (layer.mixer == LFM25_MIXER_GENERAL_DELTA ? layer.dim : layer.vdim);
}

size_t round_to(size_t value, size_t multiple) { return (value + multiple - 1) / multiple * multiple; }

// Sections of latent attention's projection start at multiples of 8 columns.
size_t latent_column(const lfm25_stack_layer& layer) { return round_to(layer.q_rank, 8); }
size_t gate_column(const lfm25_stack_layer& layer) {
    return latent_column(layer) +
           (layer.shared_cache ? 0 : round_to(static_cast<size_t>(layer.kv_rank) + layer.rot_dim, 8));
}

size_t state_space_channels(const lfm25_stack_layer& layer) {
    return static_cast<size_t>(layer.heads) * layer.vdim + 2 * static_cast<size_t>(layer.groups) * layer.state_size;
}

// Columns of the projection that the mixer reads (the matrix may have more rows, all zero).
size_t projection_columns(const lfm25_stack_layer& layer) {
    if (layer.mixer == LFM25_MIXER_ATTENTION) {
        return (static_cast<size_t>(layer.heads) + layer.kv_heads) * layer.dim +
               static_cast<size_t>(layer.kv_heads) * layer.vdim;
    }
    if (layer.mixer == LFM25_MIXER_LATENT_ATTENTION) return gate_column(layer) + mixer_columns(layer);
    if (layer.mixer == LFM25_MIXER_STATE_SPACE) return mixer_columns(layer) + state_space_channels(layer) + layer.heads;
    return 5 * static_cast<size_t>(layer.heads) * layer.dim + layer.rank;
}

const char* mixer_fault(const lfm25_stack_model& model, const lfm25_stack_layer& layer) {
    const size_t bytes = lfm25::activation_bytes(static_cast<Activation>(model.activation));
    auto convolution_fault = [&](size_t channels) -> const char* {
        if (!layer.conv || layer.conv_taps == 0) return "missing convolution";
        if (layer.conv_offset % 16 != 0 ||
            layer.conv_offset + (layer.conv_taps - 1) * channels * bytes > model.record_bytes)
            return "convolution state outside the record";
        return nullptr;
    };
    auto state_fault = [&](size_t elements) -> const char* {
        if (layer.state_offset % 16 != 0 || layer.state_offset + elements * sizeof(float) > model.record_bytes)
            return "recurrent state outside the record";
        return nullptr;
    };
    if (model.block == LFM25_BLOCK_PARALLEL) {
        const char* fault = convolution_fault(model.width);
        if (fault != nullptr) return fault;
    }
    const size_t heads = layer.heads;
    switch (layer.mixer) {
        case LFM25_MIXER_ATTENTION:
            if (layer.dim == 0 || layer.kv_heads == 0 || heads % layer.kv_heads != 0 || layer.vdim == 0)
                return "attention heads";
            if (layer.rot_dims % 2 != 0 || layer.rot_dims > layer.dim || (layer.rot_dims > 0 && !layer.inv_freq))
                return "rotary dimensions";
            if (!layer.query_norm || !layer.key_norm || !layer.key_cache || !layer.value_cache) return "attention tensors";
            return nullptr;
        case LFM25_MIXER_GENERAL_DELTA:
            if (layer.dim == 0) return "mixer without heads";
            if (layer.dim > lfm25::kDeltaMaxDim) return "delta-rule head size beyond 256";
            if (layer.rank == 0 || !layer.decay_up || !layer.decay_base || !layer.removal_bias || !layer.head_norm)
                return "delta-rule tensors";
            return state_fault(heads * layer.dim * layer.dim);
        case LFM25_MIXER_LATENT_ATTENTION:
            if (layer.dim == 0 || layer.vdim == 0 || layer.q_rank == 0 || layer.kv_rank == 0 || layer.rot_dim == 0)
                return "latent attention sizes";
            if (layer.rot_dims % 2 != 0 || layer.rot_dims > layer.rot_dim || (layer.rot_dims > 0 && !layer.inv_freq))
                return "rotary dimensions";
            if (!layer.query_latent_norm || (!layer.shared_cache && !layer.latent_norm) || !layer.key_cache ||
                !layer.value_cache || !layer.query_up.weight || !layer.latent_up.weight)
                return "latent attention tensors";
            if (layer.query_up.k != layer.q_rank || layer.query_up.n < heads * (layer.dim + layer.rot_dim) ||
                layer.latent_up.k != layer.kv_rank || layer.latent_up.n < heads * (layer.dim + layer.vdim))
                return "latent attention shapes";
            return nullptr;
        case LFM25_MIXER_STATE_SPACE: {
            if (layer.vdim == 0 || layer.groups == 0 || heads % layer.groups != 0 || layer.state_size == 0 ||
                layer.state_size > lfm25::kStateSpaceMaxSize || layer.norm_groups == 0 ||
                heads * layer.vdim % layer.norm_groups != 0)
                return "state-space sizes";
            if (!layer.conv_bias || !layer.step_bias || !layer.log_rate || !layer.skip || !layer.head_norm)
                return "state-space tensors";
            const char* fault = convolution_fault(state_space_channels(layer));
            return fault != nullptr ? fault : state_fault(heads * layer.state_size * layer.vdim);
        }
        default:
            return "unknown mixer";
    }
}

const char* layer_fault(const lfm25_stack_model& model, const lfm25_stack_layer& layer) {
    if (!layer.mixer_norm || !layer.projection.weight || !layer.output.weight) return "missing weights";
    if (layer.heads == 0) return "mixer without heads";
    const char* fault = mixer_fault(model, layer);
    if (fault != nullptr) return fault;
    if (layer.projection.k != model.width || layer.projection.n < projection_columns(layer)) return "projection shape";
    if (layer.ff_activation > LFM25_FEED_FORWARD_SQUARED_RELU) return "unknown feed-forward activation";
    const bool parallel = model.block == LFM25_BLOCK_PARALLEL;
    const size_t joined = parallel ? layer.ff : 0;
    if (layer.output.n != model.width || layer.output.k < mixer_columns(layer) + joined) return "output shape";
    if (joined == 0 && layer.output.k != mixer_columns(layer)) return "output shape";
    if (layer.ff > 0) {
        if (!layer.ff_norm || !layer.up.weight) return "missing feed-forward weights";
        if (layer.up.k != model.width || layer.up.n < layer.ff) return "up projection shape";
        if (!parallel && (!layer.down.weight || layer.down.n != model.width || layer.down.k != layer.up.n))
            return "down projection shape";
        if ((layer.ff_activation == LFM25_FEED_FORWARD_POLY_NORM) != parallel)
            return "feed-forward activation of the other arrangement";
    }
    if (!parallel && (!layer.mixer_post_norm || (layer.ff > 0 && !layer.ff_post_norm))) return "missing norms";
    return nullptr;
}

// y[m, n] = x[m, k] w[n, k]^T: tensor cores for bf16 shapes with 16-byte rows, plain f32 arithmetic otherwise.
int32_t linear(lfm25_stack_executor* self, const lfm25_stack_linear& site, const void* x, void* y, size_t rows) {
    if (self->type == Activation::kBf16 && site.k % 8 == 0 && site.n % 8 == 0) {
        lfm25_slice x_slice = {const_cast<void*>(x), rows * site.k};
        lfm25_slice w_slice = {const_cast<void*>(site.weight), site.n * site.k};
        lfm25_slice y_slice = {y, rows * site.n};
        return lfm25_blaslt_linear_bf16(self->blaslt, x_slice, w_slice, y_slice, rows, site.n, site.k);
    }
    STACK_CUDA(lfm25::launch_linear_simt(self->blaslt->stream, self->type, x, site.weight, y, rows, site.n, site.k),
               "linear launch failed");
    return LFM25_OK;
}

// One step as both batch kinds describe it.
struct Step {
    uint32_t* token_ids;
    uint32_t* positions;
    const uint32_t* request_slots;
    int64_t* physical_slots;
    const uint32_t* block_tables;
    size_t block_table_stride, block_table_rows;
    lfm25::StackSegments segments;
    const uint32_t* output_rows;   // nullptr: every token, in order
    size_t num_outputs;
    size_t decode_tokens, decode_context;   // leading single-token segments, longest context among them
    size_t prompt_context_rows;    // contexts of the other segments in whole blocks of rows, 0 = not known
    bool advance;
};

// What earlier layers of the step have left in scratch for later ones.
struct Prepared {
    const void* gathered = nullptr;    // the latent cache whose contexts lie in the context scratch
    size_t ordered = 0;                // leading tokens that token_order sorts
};

int32_t run_attention(lfm25_stack_executor* self, const Step& step, const lfm25_stack_layer& layer) {
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const lfm25::StackAttentionShape shape = {layer.heads, layer.kv_heads, layer.dim,  layer.vdim,
                                              layer.rot_dims, layer.chunk, layer.scale};
    lfm25::ProjectionNormRopeLaunch post;
    post.type = self->type;
    post.shape = shape;
    post.projected = self->projected;
    post.pitch = layer.projection.n;
    post.bias = layer.bias;
    post.query_norm = layer.query_norm;
    post.key_norm = layer.key_norm;
    post.inv_freq = layer.inv_freq;
    post.positions = step.positions;
    post.physical_slots = step.physical_slots;
    post.query_out = self->query;
    post.key_cache = layer.key_cache;
    post.value_cache = layer.value_cache;
    post.num_tokens = step.segments.num_tokens;
    post.num_pages = model.num_pages;
    post.eps = model.norm_eps;
    STACK_CUDA(lfm25::launch_projection_norm_rope(stream, post), "projection norm rope launch failed");
    lfm25::StackAttentionLaunch attention;
    attention.type = self->type;
    attention.shape = shape;
    attention.query = self->query;
    attention.key_cache = layer.key_cache;
    attention.value_cache = layer.value_cache;
    attention.block_tables = step.block_tables;
    attention.block_table_stride = step.block_table_stride;
    attention.block_table_rows = step.block_table_rows;
    attention.num_pages = model.num_pages;
    attention.request_slots = step.request_slots;
    attention.positions = step.positions;
    attention.segments = step.segments;
    attention.decode_tokens = step.decode_tokens;
    attention.decode_context = step.decode_context;
    attention.status = lfm25::device_status_words();
    attention.out = self->joined;
    attention.out_pitch = layer.output.k;
    STACK_CUDA(lfm25::launch_stack_attention(stream, attention), "attention launch failed");
    return LFM25_OK;
}

int32_t run_general_delta(lfm25_stack_executor* self, const Step& step, const lfm25_stack_layer& layer) {
    const lfm25_stack_model& model = *self->model;
    lfm25::DeltaRuleLaunch delta;
    delta.type = self->type;
    delta.segments = step.segments;
    delta.decode_tokens = step.segments.offsets != nullptr ? step.decode_tokens : 0;
    delta.heads = layer.heads;
    delta.dim = layer.dim;
    delta.rank = layer.rank;
    delta.projected = self->projected;
    delta.pitch = layer.projection.n;
    delta.decay_up = layer.decay_up;
    delta.decay_base = layer.decay_base;
    delta.removal_bias = layer.removal_bias;
    delta.norm = layer.head_norm;
    delta.record = {model.records, model.record_bytes, layer.state_offset};
    delta.raw = self->raw;
    delta.out = self->joined;
    delta.out_pitch = layer.output.k;
    delta.eps = model.norm_eps;
    STACK_CUDA(lfm25::launch_delta_rule(self->blaslt->stream, delta), "delta rule launch failed");
    return LFM25_OK;
}

// Whether the step's prompts attend to keys and values formed from their contexts' latents, instead of to the latents.
bool expands_contexts(const lfm25_stack_executor* self, const Step& step, const lfm25_stack_layer& layer) {
    const size_t prompts = step.segments.offsets != nullptr ? step.segments.num_segments - step.decode_tokens : 0;
    if (prompts == 0 || step.prompt_context_rows == 0 || step.prompt_context_rows > self->context_capacity) return false;
    if (lfm25::option(lfm25::kOptStackAttention) != 0) return false;
    if (step.segments.num_tokens - step.decode_tokens <= kShortPortion * prompts) return false;
    const lfm25::LatentAttentionShape shape = {layer.heads, layer.dim, layer.rot_dim, layer.vdim, layer.kv_rank,
                                               layer.scale};
    return lfm25::expanded_attention_supports(self->type, shape, layer.output.k, layer.projection.n, layer.latent_up.n);
}

int32_t run_latent_attention(lfm25_stack_executor* self, const Step& step, const lfm25_stack_layer& layer,
                             Prepared* prepared) {
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const size_t tokens = step.segments.num_tokens;
    const size_t bytes = lfm25::activation_bytes(self->type);
    const lfm25::LatentAttentionShape shape = {layer.heads, layer.dim, layer.rot_dim, layer.vdim, layer.kv_rank,
                                               layer.scale};
    lfm25::LatentProjectionLaunch post;
    post.type = self->type;
    post.projected = self->projected;
    post.pitch = layer.projection.n;
    post.q_rank = layer.q_rank;
    post.kv_rank = layer.kv_rank;
    post.rot_dim = layer.rot_dim;
    post.rot_dims = layer.rot_dims;
    post.latent_column = latent_column(layer);
    post.append = layer.shared_cache == 0;
    post.query_norm = layer.query_latent_norm;
    post.latent_norm = layer.latent_norm;
    post.inv_freq = layer.inv_freq;
    post.positions = step.positions;
    post.physical_slots = step.physical_slots;
    post.query_out = self->compressed;
    post.latent_cache = layer.value_cache;
    post.key_cache = layer.key_cache;
    post.num_tokens = tokens;
    post.num_pages = model.num_pages;
    post.eps = model.norm_eps;
    STACK_CUDA(lfm25::launch_latent_projection(stream, post), "latent projection launch failed");
    STACK_TRY(linear(self, layer.query_up, self->compressed, self->query, tokens));
    STACK_CUDA(lfm25::launch_rotate_queries(stream, self->type, self->query, layer.query_up.n, layer.inv_freq,
                                            step.positions, tokens, layer.heads, layer.dim, layer.rot_dim,
                                            layer.rot_dims),
               "query rotation launch failed");
    const unsigned char* gate = static_cast<const unsigned char*>(self->projected) + gate_column(layer) * bytes;
    const bool expand = expands_contexts(self, step, layer);
    const size_t direct = expand ? step.decode_tokens : tokens;      // tokens that attend to the latents
    if (direct > 0) {
        const size_t columns = static_cast<size_t>(layer.heads) * layer.kv_rank;
        lfm25::HeadLinearLaunch absorb;
        absorb.type = self->type;
        absorb.x = self->query;
        absorb.x_head = layer.dim + layer.rot_dim;
        absorb.x_pitch = layer.query_up.n;
        absorb.weight = layer.latent_up.weight;
        absorb.w_head = static_cast<size_t>(layer.dim) * layer.kv_rank;
        absorb.w_n = 1;
        absorb.w_k = layer.kv_rank;
        absorb.y = self->absorbed;
        absorb.y_pitch = columns;
        absorb.gate = nullptr;
        absorb.gate_pitch = 0;
        absorb.tokens = direct;
        absorb.n = layer.kv_rank;
        absorb.k = layer.dim;
        absorb.heads = layer.heads;
        STACK_CUDA(lfm25::launch_head_linear(stream, absorb), "query absorption launch failed");
        lfm25::LatentAttentionLaunch attention;
        attention.type = self->type;
        attention.shape = shape;
        attention.absorbed = self->absorbed;
        attention.query = self->query;
        attention.query_pitch = layer.query_up.n;
        attention.latent_cache = layer.value_cache;
        attention.key_cache = layer.key_cache;
        attention.block_tables = step.block_tables;
        attention.block_table_stride = step.block_table_stride;
        attention.block_table_rows = step.block_table_rows;
        attention.num_pages = model.num_pages;
        attention.request_slots = step.request_slots;
        attention.positions = step.positions;
        attention.token_order = nullptr;
        if (direct > 1 && direct <= lfm25::kMaxOrderTokens) {
            if (prepared->ordered != direct) {
                STACK_CUDA(lfm25::launch_context_order(stream, step.positions, direct, self->token_order),
                           "context order launch failed");
                prepared->ordered = direct;
            }
            attention.token_order = self->token_order;
        }
        attention.tokens = direct;
        attention.context = std::max(step.decode_context, direct > step.decode_tokens ? step.prompt_context_rows : 0);
        attention.status = lfm25::device_status_words();
        attention.out = self->weighted;
        STACK_CUDA(lfm25::launch_latent_attention(stream, attention), "latent attention launch failed");
        lfm25::HeadLinearLaunch value = absorb;
        value.x = self->weighted;
        value.x_pitch = columns;
        value.x_head = layer.kv_rank;
        value.weight = static_cast<const unsigned char*>(layer.latent_up.weight) +
                       static_cast<size_t>(layer.heads) * layer.dim * layer.kv_rank * 2;
        value.w_head = static_cast<size_t>(layer.vdim) * layer.kv_rank;
        value.w_n = layer.kv_rank;
        value.w_k = 1;
        value.y = self->joined;
        value.y_pitch = layer.output.k;
        value.gate = gate;
        value.gate_pitch = layer.projection.n;
        value.n = layer.vdim;
        value.k = layer.kv_rank;
        STACK_CUDA(lfm25::launch_head_linear(stream, value), "value projection launch failed");
    }
    if (!expand) return LFM25_OK;
    const size_t rows = step.prompt_context_rows;
    if (prepared->gathered != layer.value_cache) {
        if (prepared->gathered == nullptr) {
            STACK_CUDA(lfm25::launch_context_bases(stream, step.segments, step.positions, step.decode_tokens,
                                                   self->context_bases),
                       "context layout launch failed");
        }
        lfm25::GatherContextLaunch gather;
        gather.type = self->type;
        gather.segments = step.segments;
        gather.first_segment = step.decode_tokens;
        gather.bases = self->context_bases;
        gather.positions = step.positions;
        gather.block_tables = step.block_tables;
        gather.block_table_stride = step.block_table_stride;
        gather.block_table_rows = step.block_table_rows;
        gather.num_pages = model.num_pages;
        gather.kv_rank = layer.kv_rank;
        gather.rot_dim = layer.rot_dim;
        gather.latent_cache = layer.value_cache;
        gather.key_cache = layer.key_cache;
        gather.latents = self->context_latents;
        gather.keys = self->context_keys;
        gather.rows = rows;
        STACK_CUDA(lfm25::launch_gather_context(stream, gather), "context gather launch failed");
        prepared->gathered = layer.value_cache;
    }
    STACK_TRY(linear(self, layer.latent_up, self->context_latents, self->expanded, rows));
    lfm25::ExpandedAttentionLaunch attention;
    attention.type = self->type;
    attention.shape = shape;
    attention.query = self->query;
    attention.query_pitch = layer.query_up.n;
    attention.expanded = self->expanded;
    attention.expanded_pitch = layer.latent_up.n;
    attention.keys = self->context_keys;
    attention.bases = self->context_bases;
    attention.rows = rows;
    attention.first_segment = step.decode_tokens;
    attention.segments = step.segments;
    attention.positions = step.positions;
    attention.gate = gate;
    attention.gate_pitch = layer.projection.n;
    attention.status = lfm25::device_status_words();
    attention.out = self->joined;
    attention.out_pitch = layer.output.k;
    STACK_CUDA(lfm25::launch_expanded_attention(stream, attention), "prompt attention launch failed");
    return LFM25_OK;
}

int32_t run_state_space(lfm25_stack_executor* self, const Step& step, const lfm25_stack_layer& layer) {
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const size_t bytes = lfm25::activation_bytes(self->type);
    const size_t inner = mixer_columns(layer), channels = state_space_channels(layer);
    const unsigned char* projected = static_cast<const unsigned char*>(self->projected);
    lfm25::ChannelConvLaunch conv;
    conv.type = self->type;
    conv.segments = step.segments;
    conv.x = projected + inner * bytes;
    conv.pitch = layer.projection.n;
    conv.conv = layer.conv;
    conv.bias = layer.conv_bias;
    conv.taps = layer.conv_taps;
    conv.record = {model.records, model.record_bytes, layer.conv_offset};
    conv.out = self->convolved;
    conv.channels = channels;
    STACK_CUDA(lfm25::launch_channel_conv(stream, conv), "channel convolution launch failed");
    lfm25::StateSpaceLaunch scan;
    scan.type = self->type;
    scan.segments = step.segments;
    scan.decode_tokens = step.decode_tokens;
    scan.heads = layer.heads;
    scan.groups = layer.groups;
    scan.size = layer.state_size;
    scan.vdim = layer.vdim;
    scan.mixed = self->convolved;
    scan.mixed_pitch = channels;
    scan.raw_step = projected + (inner + channels) * bytes;
    scan.step_pitch = layer.projection.n;
    scan.step_bias = layer.step_bias;
    scan.log_rate = layer.log_rate;
    scan.skip = layer.skip;
    scan.record = {model.records, model.record_bytes, layer.state_offset};
    scan.out = self->scanned;
    STACK_CUDA(lfm25::launch_state_space(stream, scan), "state-space launch failed");
    lfm25::GatedGroupNormLaunch norm;
    norm.type = self->type;
    norm.y = self->scanned;
    norm.z = projected;
    norm.z_pitch = layer.projection.n;
    norm.norm = layer.head_norm;
    norm.out = self->joined;
    norm.out_pitch = layer.output.k;
    norm.tokens = step.segments.num_tokens;
    norm.width = inner;
    norm.groups = layer.norm_groups;
    norm.eps = model.norm_eps;
    STACK_CUDA(lfm25::launch_gated_group_norm(stream, norm), "gated norm launch failed");
    return LFM25_OK;
}

int32_t run_mixer(lfm25_stack_executor* self, const Step& step, const lfm25_stack_layer& layer, Prepared* prepared) {
    STACK_TRY(linear(self, layer.projection, self->mixed, self->projected, step.segments.num_tokens));
    switch (layer.mixer) {
        case LFM25_MIXER_ATTENTION: return run_attention(self, step, layer);
        case LFM25_MIXER_GENERAL_DELTA: return run_general_delta(self, step, layer);
        case LFM25_MIXER_LATENT_ATTENTION: return run_latent_attention(self, step, layer, prepared);
        default: return run_state_space(self, step, layer);
    }
}

int32_t enqueue_parallel(lfm25_stack_executor* self, const Step& step) {
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const size_t tokens = step.segments.num_tokens;
    Prepared prepared;
    int current = 0;
    for (uint32_t index = 0; index < self->depth; ++index) {
        const lfm25_stack_layer& layer = model.layers[index];
        lfm25::ResidualNormConvLaunch head;
        head.type = self->type;
        head.segments = step.segments;
        head.residual = self->residual[current];
        head.update = index == 0 ? nullptr : self->update;
        head.token_ids = step.token_ids;
        head.embedding = index == 0 ? model.embedding : nullptr;
        head.vocab = model.vocab;
        head.mixer_norm = layer.mixer_norm;
        head.ff_norm = layer.ff > 0 ? layer.ff_norm : nullptr;
        head.conv = layer.conv;
        head.taps = layer.conv_taps;
        head.record = {model.records, model.record_bytes, layer.conv_offset};
        head.residual_out = self->residual[1 - current];
        head.mixed_out = self->mixed;
        head.ff_out = self->normalized;
        head.width = model.width;
        head.eps = model.norm_eps;
        STACK_CUDA(lfm25::launch_residual_norm_conv(stream, head), "residual norm convolution launch failed");
        current = 1 - current;
        STACK_TRY(run_mixer(self, step, layer, &prepared));
        if (layer.ff > 0) {
            STACK_TRY(linear(self, layer.up, self->normalized, self->up, tokens));
            const size_t column = mixer_columns(layer);
            unsigned char* activation =
                static_cast<unsigned char*>(self->joined) + column * lfm25::activation_bytes(self->type);
            STACK_CUDA(lfm25::launch_poly_norm(stream, self->type, self->up, layer.up.n, activation, layer.output.k,
                                               tokens, layer.ff, layer.output.k - column - layer.ff, layer.poly,
                                               model.norm_eps),
                       "polynomial activation launch failed");
        }
        STACK_TRY(linear(self, layer.output, self->joined, self->update, tokens));
    }
    self->last_residual = self->residual[current];
    self->last_post = nullptr;
    if (step.num_outputs == 0) return LFM25_OK;
    STACK_CUDA(lfm25::launch_residual_norm_rows(stream, self->type, self->residual[current], self->update,
                                                model.final_norm, step.output_rows, self->head_input, step.num_outputs,
                                                tokens, model.width, model.norm_eps),
               "final norm launch failed");
    return LFM25_OK;
}

int32_t enqueue_sandwich(lfm25_stack_executor* self, const Step& step) {
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const size_t tokens = step.segments.num_tokens;
    Prepared prepared;
    lfm25::ResidualPostNormLaunch norm;
    norm.type = self->type;
    norm.residual = self->residual[0];
    norm.update = nullptr;
    norm.post_norm = nullptr;
    norm.token_ids = step.token_ids;
    norm.embedding = model.embedding;
    norm.vocab = model.vocab;
    norm.rows = nullptr;
    norm.residual_out = self->residual[0];
    norm.num_rows = tokens;
    norm.num_tokens = tokens;
    norm.width = model.width;
    norm.shift = model.norm_shift;
    norm.eps = model.norm_eps;
    // x <- x + N(update of the sublayer before), then the norm in front of the next one
    auto enter = [&](const void* weight, void* out) -> int32_t {
        norm.norm = weight;
        norm.out = out;
        STACK_CUDA(lfm25::launch_residual_post_norm(stream, norm), "residual norm launch failed");
        norm.embedding = nullptr;
        norm.update = self->update;
        return LFM25_OK;
    };
    for (uint32_t index = 0; index < self->depth; ++index) {
        const lfm25_stack_layer& layer = model.layers[index];
        STACK_TRY(enter(layer.mixer_norm, self->mixed));
        STACK_TRY(run_mixer(self, step, layer, &prepared));
        STACK_TRY(linear(self, layer.output, self->joined, self->update, tokens));
        norm.post_norm = layer.mixer_post_norm;
        if (layer.ff > 0) {
            STACK_TRY(enter(layer.ff_norm, self->normalized));
            STACK_TRY(linear(self, layer.up, self->normalized, self->up, tokens));
            STACK_CUDA(lfm25::launch_squared_relu(stream, self->type, self->up, tokens * layer.up.n),
                       "activation launch failed");
            STACK_TRY(linear(self, layer.down, self->up, self->update, tokens));
            norm.post_norm = layer.ff_post_norm;
        }
    }
    self->last_residual = self->residual[0];
    self->last_post = norm.post_norm;
    if (step.num_outputs == 0) return LFM25_OK;
    norm.rows = step.output_rows;
    norm.num_rows = step.num_outputs;
    norm.residual_out = nullptr;
    return enter(model.final_norm, self->head_input);
}

int32_t enqueue(lfm25_stack_executor* self, const Step& step) {
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const size_t tokens = step.segments.num_tokens;
    STACK_CUDA(lfm25::launch_decode_metadata(stream, step.token_ids, step.positions, step.request_slots,
                                             step.block_tables, self->sampled, step.physical_slots, tokens,
                                             step.block_table_stride, step.block_table_rows, model.num_pages,
                                             step.advance),
               "step metadata launch failed");
    self->last_tokens = tokens;
    STACK_TRY(model.block == LFM25_BLOCK_PARALLEL ? enqueue_parallel(self, step) : enqueue_sandwich(self, step));
    if (step.num_outputs == 0) {
        return LFM25_OK;
    }
    STACK_TRY(linear(self, model.head, self->head_input, self->logits, step.num_outputs));
    STACK_CUDA(lfm25::launch_argmax_rows(stream, self->type, self->logits, model.head.n, self->sampled, step.num_outputs,
                                         model.vocab),
               "argmax launch failed");
    return LFM25_OK;
}

uint64_t signature(const lfm25_stack_executor* self, const lfm25_decode_batch* batch) {
    lfm25::Fnv1a hash;
    hash.add(batch->token_ids);
    hash.add(batch->positions);
    hash.add(batch->request_slots);
    hash.add(batch->physical_slots);
    hash.add(batch->block_tables);
    hash.add(batch->block_table_stride);
    hash.add(batch->block_table_rows);
    hash.add(self->depth);
    const lfm25_stack_model& model = *self->model;
    hash.add(model.layers);
    hash.add(model.embedding);
    hash.add(model.final_norm);
    hash.add(model.head.weight);
    hash.add(model.head.n);
    hash.add(model.vocab);
    hash.add(model.width);
    hash.add(model.norm_eps);
    hash.add(model.norm_shift);
    hash.add(model.logit_softcap);
    hash.add(model.block);
    hash.add(model.records);
    hash.add(model.record_bytes);
    hash.add(model.num_request_slots);
    hash.add(model.num_pages);
    for (uint32_t index = 0; index < model.num_layers; ++index) {
        const lfm25_stack_layer& layer = model.layers[index];
        const void* pointers[] = {layer.mixer_norm, layer.ff_norm, layer.conv, layer.projection.weight, layer.output.weight,
                                  layer.up.weight, layer.inv_freq, layer.bias, layer.query_norm, layer.key_norm,
                                  layer.key_cache, layer.value_cache, layer.decay_up, layer.decay_base,
                                  layer.removal_bias, layer.head_norm, layer.down.weight, layer.mixer_post_norm,
                                  layer.ff_post_norm, layer.query_latent_norm, layer.latent_norm, layer.query_up.weight,
                                  layer.latent_up.weight, layer.conv_bias, layer.step_bias, layer.log_rate, layer.skip};
        for (const void* pointer : pointers) hash.add(pointer);
        const size_t sizes[] = {layer.conv_offset, layer.projection.n, layer.output.k, layer.up.n, layer.state_offset,
                                layer.down.k, layer.query_up.n, layer.latent_up.n};
        for (size_t size : sizes) hash.add(size);
        const uint32_t words[] = {layer.mixer, layer.ff, layer.heads, layer.dim, layer.kv_heads, layer.vdim,
                                  layer.rot_dims, layer.chunk, layer.rank, layer.conv_taps, layer.ff_activation,
                                  layer.q_rank, layer.kv_rank, layer.rot_dim, layer.shared_cache, layer.groups,
                                  layer.state_size, layer.norm_groups};
        for (uint32_t word : words) hash.add(word);
        for (float value : layer.poly) hash.add(value);
        hash.add(layer.scale);
    }
    for (int which = 0; which < lfm25::kOptCount; ++which) {
        if (which != lfm25::kOptEngineGraph) hash.add(lfm25::option(static_cast<lfm25::Option>(which)));
    }
    hash.add(self->blaslt->tuning_kernel);
    hash.add(self->blaslt->tuning);
    hash.add(self->blaslt->stream);
    return hash.state;
}

int32_t decode_step(const lfm25_stack_executor* self, const lfm25_decode_batch* batch, bool advance, Step* step) {
    if (self == nullptr || batch == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "stack executor received a null argument");
    }
    if (batch->num_tokens == 0 || batch->num_tokens > self->maximum_tokens || batch->num_tokens > self->maximum_rows) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "stack executor token count exceeds workspace");
    }
    if (!batch->token_ids || !batch->positions || !batch->request_slots || !batch->physical_slots ||
        !batch->block_tables || batch->block_table_stride == 0 || batch->block_table_rows == 0) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "decode batch metadata is incomplete");
    }
    step->token_ids = batch->token_ids;
    step->positions = batch->positions;
    step->request_slots = batch->request_slots;
    step->physical_slots = batch->physical_slots;
    step->block_tables = batch->block_tables;
    step->block_table_stride = batch->block_table_stride;
    step->block_table_rows = batch->block_table_rows;
    step->segments = {nullptr, batch->request_slots, batch->num_tokens, batch->num_tokens, self->model->num_request_slots};
    step->output_rows = nullptr;
    step->num_outputs = batch->num_tokens;
    step->decode_tokens = batch->num_tokens;
    // rounded up to a power of two: the context decides how the decode attention splits the keys, and a captured step
    // serves every context of its class
    step->decode_context = 1;
    while (step->decode_context < batch->max_context_tokens) step->decode_context *= 2;
    step->prompt_context_rows = 0;
    step->advance = advance;
    return LFM25_OK;
}

}  // namespace

extern "C" {

int32_t lfm25_stack_executor_create(lfm25_blaslt* blaslt, const lfm25_stack_model* model, size_t maximum_tokens,
                                    size_t maximum_rows, lfm25_stack_executor** out) {
    if (blaslt == nullptr || model == nullptr || out == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "stack executor received a null argument");
    }
    if (maximum_rows == 0 || maximum_tokens < maximum_rows || maximum_tokens > 65536) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT,
                                   "stack executor needs 1..=65536 tokens per step and at most as many output rows");
    }
    if (model->num_layers == 0 || model->layers == nullptr || model->embedding == nullptr ||
        model->final_norm == nullptr || model->head.weight == nullptr || model->records == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "stack model is incomplete");
    }
    if (model->activation > LFM25_ACTIVATION_F32 || model->block > LFM25_BLOCK_SANDWICH || model->width == 0 ||
        model->vocab == 0 || model->head.n < model->vocab || model->head.k != model->width || model->record_bytes % 256 != 0 ||
        model->num_request_slots == 0 || model->num_pages == 0) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "stack model sizes are inconsistent");
    }
    size_t projection = 0, query = 0, up = 0, joined = 0, raw = 0, compressed = 0, latents = 0, channels = 0, scanned = 0;
    size_t context_rank = 0, context_keys = 0, context_columns = 0;
    const Activation type = static_cast<Activation>(model->activation);
    for (uint32_t index = 0; index < model->num_layers; ++index) {
        const lfm25_stack_layer& layer = model->layers[index];
        const char* fault = layer_fault(*model, layer);
        if (fault != nullptr) {
            char message[120];
            snprintf(message, sizeof message, "layer %u: %s", index, fault);
            return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, message);
        }
        projection = std::max(projection, layer.projection.n);
        joined = std::max(joined, layer.output.k);
        up = std::max(up, layer.ff > 0 ? layer.up.n : 0);
        const size_t width = static_cast<size_t>(layer.heads) * layer.dim;
        if (layer.mixer == LFM25_MIXER_ATTENTION) query = std::max(query, width);
        if (layer.mixer == LFM25_MIXER_GENERAL_DELTA && lfm25::delta_rule_needs_scratch(layer.dim))
            raw = std::max(raw, width);
        if (layer.mixer == LFM25_MIXER_LATENT_ATTENTION) {
            const lfm25::LatentAttentionShape shape = {layer.heads, layer.dim, layer.rot_dim, layer.vdim, layer.kv_rank,
                                                       layer.scale};
            compressed = std::max<size_t>(compressed, layer.q_rank);
            query = std::max(query, layer.query_up.n);
            latents = std::max(latents, static_cast<size_t>(layer.heads) * layer.kv_rank);
            if (lfm25::expanded_attention_supports(type, shape, layer.output.k, layer.projection.n, layer.latent_up.n)) {
                context_rank = std::max<size_t>(context_rank, layer.kv_rank);
                context_keys = std::max<size_t>(context_keys, layer.rot_dim);
                context_columns = std::max(context_columns, layer.latent_up.n);
            }
        }
        if (layer.mixer == LFM25_MIXER_STATE_SPACE) {
            channels = std::max(channels, state_space_channels(layer));
            scanned = std::max(scanned, mixer_columns(layer));
        }
    }
    lfm25_stack_executor* self = new (std::nothrow) lfm25_stack_executor();
    if (self == nullptr) return lfm25::report_error(LFM25_ERR_CUDA, "out of host memory");
    self->blaslt = blaslt;
    self->model = model;
    self->type = type;
    self->maximum_tokens = maximum_tokens;
    self->maximum_rows = maximum_rows;
    self->depth = model->num_layers;
    const size_t t = maximum_tokens, r = maximum_rows, bytes = lfm25::activation_bytes(self->type);
    size_t c = 0;
    if (context_columns > 0) {
        // every segment may leave part of its last block of rows unused
        const size_t wanted = std::max<size_t>(4 * t, model->num_pages * 16) + r * LFM25_CONTEXT_ROWS;
        c = std::max<size_t>(1, std::min(wanted, kContextBytes / (context_columns * bytes)) / LFM25_CONTEXT_ROWS) *
            LFM25_CONTEXT_ROWS;
    }
    self->context_capacity = c;
    void** fields[] = {reinterpret_cast<void**>(&self->residual[0]), reinterpret_cast<void**>(&self->residual[1]),
                       &self->mixed, &self->normalized, &self->projected, &self->query, &self->up, &self->joined,
                       &self->update, &self->head_input, &self->logits, reinterpret_cast<void**>(&self->raw),
                       reinterpret_cast<void**>(&self->sampled), &self->compressed, &self->absorbed, &self->weighted,
                       &self->context_latents, &self->context_keys, &self->expanded,
                       reinterpret_cast<void**>(&self->context_bases), reinterpret_cast<void**>(&self->token_order),
                       &self->convolved, &self->scanned};
    const size_t sizes[] = {t * model->width * 4, t * model->width * 4, t * model->width * bytes,
                            t * model->width * bytes, t * projection * bytes, t * query * bytes, t * up * bytes,
                            t * joined * bytes, t * model->width * bytes, r * model->width * bytes,
                            r * model->head.n * bytes, t * raw * 4, r * 4, t * compressed * bytes, t * latents * bytes,
                            t * latents * bytes, c * context_rank * bytes, c * context_keys * bytes,
                            c * context_columns * bytes, (t + 1) * 4, latents > 0 ? t * 4 : 0, t * channels * bytes,
                            t * scanned * bytes};
    size_t total = 0;
    for (size_t size : sizes) total += (size + 255) & ~static_cast<size_t>(255);
    cudaError_t status = cudaMalloc(&self->allocation, total);
    if (status == cudaSuccess) status = cudaMemsetAsync(self->allocation, 0, total, blaslt->stream);
    if (status != cudaSuccess) {
        cudaFree(self->allocation);
        delete self;
        return cuda_failure(status, "failed to allocate stack scratch");
    }
    unsigned char* cursor = static_cast<unsigned char*>(self->allocation);
    for (size_t index = 0; index < sizeof sizes / sizeof sizes[0]; ++index) {
        *fields[index] = sizes[index] > 0 ? cursor : nullptr;
        cursor += (sizes[index] + 255) & ~static_cast<size_t>(255);
    }
    *out = self;
    return LFM25_OK;
}

void lfm25_stack_executor_destroy(lfm25_stack_executor* self) {
    if (self == nullptr) return;
    cudaFree(self->allocation);
    cudaFree(self->exported);
    delete self;
}

int32_t lfm25_stack_executor_forward(lfm25_stack_executor* self, const lfm25_decode_batch* batch, uint32_t advance) {
    Step step;
    STACK_TRY(decode_step(self, batch, advance != 0, &step));
    return enqueue(self, step);
}

int32_t lfm25_stack_executor_step_graph(lfm25_stack_executor* self, const lfm25_decode_batch* batch, uint32_t advance) {
    Step step;
    STACK_TRY(decode_step(self, batch, advance != 0, &step));
    lfm25::StepKey key;
    key.num_tokens = batch->num_tokens;
    key.splits = step.decode_context;
    key.flags = advance != 0 ? 1u : 0u;
    key.signature = signature(self, batch);
    return self->graphs.run(key, self->blaslt->stream, [&]() -> int32_t { return enqueue(self, step); });
}

int32_t lfm25_stack_executor_forward_ragged(lfm25_stack_executor* self, const lfm25_ragged_batch* batch,
                                            size_t num_output_rows) {
    if (self == nullptr || batch == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "stack executor received a null argument");
    }
    if (batch->num_tokens == 0 || batch->num_tokens > self->maximum_tokens || num_output_rows > self->maximum_rows ||
        batch->num_segments == 0 || batch->num_segments > batch->num_tokens ||
        batch->num_decode_segments > batch->num_segments) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "ragged step exceeds the stack executor's workspace");
    }
    if (!batch->token_ids || !batch->positions || !batch->request_slots || !batch->physical_slots ||
        !batch->segment_offsets || !batch->segment_slots || (num_output_rows > 0 && !batch->output_rows) ||
        !batch->block_tables || batch->block_table_stride == 0 || batch->block_table_rows == 0) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "ragged batch metadata is incomplete");
    }
    Step step;
    step.token_ids = const_cast<uint32_t*>(batch->token_ids);
    step.positions = const_cast<uint32_t*>(batch->positions);
    step.request_slots = batch->request_slots;
    step.physical_slots = batch->physical_slots;
    step.block_tables = batch->block_tables;
    step.block_table_stride = batch->block_table_stride;
    step.block_table_rows = batch->block_table_rows;
    step.segments = {batch->segment_offsets, batch->segment_slots, batch->num_segments, batch->num_tokens,
                     self->model->num_request_slots};
    step.output_rows = batch->output_rows;
    step.num_outputs = num_output_rows;
    step.decode_tokens = batch->num_decode_segments;
    step.decode_context = batch->max_decode_context_tokens;
    step.prompt_context_rows = batch->prompt_context_rows;
    step.advance = false;
    return enqueue(self, step);
}

int32_t lfm25_stack_executor_download_sampled(lfm25_stack_executor* self, uint32_t* host, size_t count) {
    if (self == nullptr || host == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "sampled download received a null argument");
    }
    if (count > self->maximum_rows) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "sampled download exceeds the executor's capacity");
    }
    STACK_CUDA(cudaMemcpyAsync(host, self->sampled, count * sizeof(uint32_t), cudaMemcpyDeviceToHost,
                               self->blaslt->stream),
               "sampled download failed");
    return LFM25_OK;
}

int32_t lfm25_stack_executor_read_logits(lfm25_stack_executor* self, float* host, size_t rows) {
    if (self == nullptr || host == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "logits read received a null argument");
    }
    if (rows > self->maximum_rows) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "logits read exceeds the executor's capacity");
    }
    const lfm25_stack_model& model = *self->model;
    cudaStream_t stream = self->blaslt->stream;
    const size_t bytes = rows * model.vocab * sizeof(float);
    if (bytes == 0) return LFM25_OK;
    if (bytes > self->exported_bytes) {
        cudaFree(self->exported);
        self->exported = nullptr;
        self->exported_bytes = 0;
        STACK_CUDA(cudaMalloc(reinterpret_cast<void**>(&self->exported), bytes), "failed to allocate logits for export");
        self->exported_bytes = bytes;
    }
    STACK_CUDA(lfm25::launch_export_logits(stream, self->type, self->logits, model.head.n, self->exported, rows, model.vocab,
                                           model.logit_softcap),
               "logits export launch failed");
    STACK_CUDA(cudaMemcpyAsync(host, self->exported, bytes, cudaMemcpyDeviceToHost, stream), "logits download failed");
    STACK_CUDA(cudaStreamSynchronize(stream), "logits download failed");
    return LFM25_OK;
}

int32_t lfm25_stack_executor_set_depth(lfm25_stack_executor* self, uint32_t layers) {
    if (self == nullptr) return lfm25::report_error(LFM25_ERR_NULL_POINTER, "stack executor is null");
    if (layers > self->model->num_layers) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "depth exceeds the model's layers");
    }
    self->depth = layers == 0 ? self->model->num_layers : layers;
    return LFM25_OK;
}

int32_t lfm25_stack_executor_read_residual(lfm25_stack_executor* self, float* host, size_t tokens) {
    if (self == nullptr || host == nullptr) {
        return lfm25::report_error(LFM25_ERR_NULL_POINTER, "residual read received a null argument");
    }
    if (tokens == 0 || tokens > self->last_tokens) {
        return lfm25::report_error(LFM25_ERR_INVALID_ARGUMENT, "residual read exceeds the last step");
    }
    const size_t count = tokens * self->model->width;
    const size_t bytes = lfm25::activation_bytes(self->type);
    cudaStream_t stream = self->blaslt->stream;
    if (self->last_post != nullptr) {
        lfm25::ResidualPostNormLaunch norm = {};
        norm.type = self->type;
        norm.residual = self->last_residual;
        norm.update = self->update;
        norm.post_norm = self->last_post;
        norm.residual_out = self->residual[1];
        norm.num_rows = tokens;
        norm.num_tokens = tokens;
        norm.width = self->model->width;
        norm.shift = self->model->norm_shift;
        norm.eps = self->model->norm_eps;
        STACK_CUDA(lfm25::launch_residual_post_norm(stream, norm), "residual norm launch failed");
        STACK_CUDA(cudaMemcpyAsync(host, self->residual[1], count * 4, cudaMemcpyDeviceToHost, stream),
                   "residual download failed");
        STACK_CUDA(cudaStreamSynchronize(stream), "residual download failed");
        return LFM25_OK;
    }
    self->staging.resize(count * bytes);
    STACK_CUDA(cudaMemcpyAsync(host, self->last_residual, count * 4, cudaMemcpyDeviceToHost, stream),
               "residual download failed");
    STACK_CUDA(cudaMemcpyAsync(self->staging.data(), self->update, count * bytes, cudaMemcpyDeviceToHost, stream),
               "residual download failed");
    STACK_CUDA(cudaStreamSynchronize(stream), "residual download failed");
    for (size_t index = 0; index < count; ++index) {
        float add;
        if (self->type == Activation::kF32) {
            memcpy(&add, self->staging.data() + index * 4, 4);
        } else {
            uint16_t half;
            memcpy(&half, self->staging.data() + index * 2, 2);
            const uint32_t word = static_cast<uint32_t>(half) << 16;
            memcpy(&add, &word, 4);
        }
        host[index] += add;
    }
    return LFM25_OK;
}

size_t lfm25_stack_executor_graph_kernels(const lfm25_stack_executor* self) {
    return self != nullptr ? self->graphs.last_kernel_nodes() : 0;
}

size_t lfm25_stack_executor_graph_captures(const lfm25_stack_executor* self) {
    return self != nullptr ? self->graphs.captures() : 0;
}

}  // extern "C"
