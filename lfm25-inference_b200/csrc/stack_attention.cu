// Attention of the layer stack for any number of heads, head sizes and chunk length: projection biases, norms over the
// whole query and key projections, rotary positions and the paged append in one kernel, and attention over the paged
// cache with scores, softmax and weights in 32 bits.
#include <math.h>

#include "launch.h"
#include "options.h"
#include "stack_attention.h"
#include "stack_common.cuh"

namespace lfm25 {

namespace {

constexpr uint32_t kPostThreads = 256;

template <typename T>
struct PostArgs {
    StackAttentionShape shape;
    const T* projected;
    size_t pitch;
    const __nv_bfloat16* bias;
    const __nv_bfloat16* query_norm;
    const __nv_bfloat16* key_norm;
    const float* inv_freq;
    const uint32_t* positions;
    const int64_t* physical_slots;
    T* query_out;
    T* key_cache;
    T* value_cache;
    size_t num_pages;
    float eps;
};

template <typename T, int VEC>
__device__ __forceinline__ void biased(const PostArgs<T>& args, const T* row, size_t column, float (&value)[VEC]) {
    load_values<VEC>(row + column, value);
    if (args.bias != nullptr) {
        float bias[VEC];
        load_values<VEC>(args.bias + column, bias);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] += bias[i];
    }
}

// One value vector of a normalised and rotated head: dimension `i` .. `i + VEC - 1` of the head that starts at
// `head_column` of the row.
template <typename T, int VEC>
__device__ __forceinline__ void rotated(const PostArgs<T>& args, const T* row, const __nv_bfloat16* norm,
                                        size_t section, size_t head_column, uint32_t i, float scale,
                                        const float2* angles, float (&value)[VEC]) {
    float weight[VEC];
    biased<T, VEC>(args, row, section + head_column + i, value);
    load_values<VEC>(norm + head_column + i, weight);
#pragma unroll
    for (int e = 0; e < VEC; ++e) value[e] *= scale * weight[e];
    if (i >= args.shape.rot_dims) {
        return;
    }
    const uint32_t half = args.shape.rot_dims / 2;
    const bool first = i < half;
    const uint32_t partner = first ? i + half : i - half;
    float other[VEC];
    biased<T, VEC>(args, row, section + head_column + partner, other);
    load_values<VEC>(norm + head_column + partner, weight);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        other[e] *= scale * weight[e];
        const float2 angle = angles[(first ? i : partner) + e];      // (cos, sin)
        value[e] = first ? value[e] * angle.x - other[e] * angle.y : value[e] * angle.x + other[e] * angle.y;
    }
}

// One CTA per token.  The two row norms run over all heads at once, so the sums come first; every output vector is then
// formed from the projection again (L1-resident) together with its rotation partner.
template <typename T, int VEC>
__global__ void __launch_bounds__(kPostThreads)
projection_norm_rope_kernel(const PostArgs<T> args) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float2 angles[];                // [rot_dims / 2] (cos, sin)
    __shared__ float scratch[2][kPostThreads / 32];
    const StackAttentionShape& shape = args.shape;
    const size_t token = blockIdx.x;
    const T* row = args.projected + token * args.pitch;
    const size_t query_width = static_cast<size_t>(shape.heads) * shape.dim;
    const size_t key_width = static_cast<size_t>(shape.kv_heads) * shape.dim;
    const size_t value_width = static_cast<size_t>(shape.kv_heads) * shape.vdim;
    const float position = static_cast<float>(args.positions[token]);
    for (uint32_t i = threadIdx.x; i < shape.rot_dims / 2; i += kPostThreads) {
        float sine, cosine;
        sincosf(position * args.inv_freq[i], &sine, &cosine);
        angles[i] = make_float2(cosine, sine);
    }
    float query_sum = 0.0f, key_sum = 0.0f;
    for (size_t column = threadIdx.x * VEC; column < query_width + key_width; column += kPostThreads * VEC) {
        float value[VEC], sum = 0.0f;
        biased<T, VEC>(args, row, column, value);
#pragma unroll
        for (int e = 0; e < VEC; ++e) sum = fmaf(value[e], value[e], sum);
        if (column < query_width) {
            query_sum += sum;
        } else {
            key_sum += sum;
        }
    }
    query_sum = warp_sum(query_sum);
    key_sum = warp_sum(key_sum);
    const uint32_t lane = threadIdx.x & 31;
    if (lane == 0) {
        scratch[0][threadIdx.x >> 5] = query_sum;
        scratch[1][threadIdx.x >> 5] = key_sum;
    }
    __syncthreads();
    query_sum = warp_sum(lane < kPostThreads / 32 ? scratch[0][lane] : 0.0f);
    key_sum = warp_sum(lane < kPostThreads / 32 ? scratch[1][lane] : 0.0f);
    const float query_scale = inverse_rms(query_sum, query_width, args.eps);
    const float key_scale = inverse_rms(key_sum, key_width, args.eps);

    for (size_t column = threadIdx.x * VEC; column < query_width; column += kPostThreads * VEC) {
        const uint32_t i = static_cast<uint32_t>(column % shape.dim);
        float value[VEC];
        rotated<T, VEC>(args, row, args.query_norm, 0, column - i, i, query_scale, angles, value);
        store_values<VEC>(args.query_out + token * query_width + column, value);
    }
    const int64_t slot = args.physical_slots[token];
    const size_t page = slot < 0 ? args.num_pages : static_cast<size_t>(slot) / kPageSize;
    if (page >= args.num_pages) {
        return;
    }
    const size_t offset = static_cast<size_t>(slot) % kPageSize;
    for (size_t column = threadIdx.x * VEC; column < key_width; column += kPostThreads * VEC) {
        const uint32_t i = static_cast<uint32_t>(column % shape.dim);
        const size_t head = column / shape.dim;
        float value[VEC];
        rotated<T, VEC>(args, row, args.key_norm, query_width, column - i, i, key_scale, angles, value);
        store_values<VEC>(args.key_cache + ((page * shape.kv_heads + head) * kPageSize + offset) * shape.dim + i, value);
    }
    for (size_t column = threadIdx.x * VEC; column < value_width; column += kPostThreads * VEC) {
        const size_t head = column / shape.vdim;
        float value[VEC];
        biased<T, VEC>(args, row, query_width + key_width + column, value);
        store_values<VEC>(args.value_cache + ((page * shape.kv_heads + head) * kPageSize + offset) * shape.vdim +
                              column % shape.vdim,
                          value);
    }
}

template <typename T>
cudaError_t launch_post(cudaStream_t stream, const ProjectionNormRopeLaunch& launch) {
    PostArgs<T> args;
    args.shape = launch.shape;
    args.projected = static_cast<const T*>(launch.projected);
    args.pitch = launch.pitch;
    args.bias = static_cast<const __nv_bfloat16*>(launch.bias);
    args.query_norm = static_cast<const __nv_bfloat16*>(launch.query_norm);
    args.key_norm = static_cast<const __nv_bfloat16*>(launch.key_norm);
    args.inv_freq = launch.inv_freq;
    args.positions = launch.positions;
    args.physical_slots = launch.physical_slots;
    args.query_out = static_cast<T*>(launch.query_out);
    args.key_cache = static_cast<T*>(launch.key_cache);
    args.value_cache = static_cast<T*>(launch.value_cache);
    args.num_pages = launch.num_pages;
    args.eps = launch.eps;
    const bool vector = launch.shape.dim % 8 == 0 && launch.shape.vdim % 8 == 0 && launch.shape.rot_dims % 16 == 0 &&
                        launch.pitch % 8 == 0 && aligned_to(launch.projected, 16) && aligned_to(launch.bias, 16) &&
                        aligned_to(launch.query_norm, 16) && aligned_to(launch.key_norm, 16) &&
                        aligned_to(launch.query_out, 16) && aligned_to(launch.key_cache, 16) &&
                        aligned_to(launch.value_cache, 16);
    return launch_kernel(vector ? projection_norm_rope_kernel<T, 8> : projection_norm_rope_kernel<T, 1>,
                         static_cast<unsigned int>(launch.num_tokens), kPostThreads,
                         launch.shape.rot_dims / 2 * sizeof(float2), stream, 1, args);
}

// ---------------------------------------------------------------------------------------- scalar attention kernel

constexpr uint32_t kScalarThreads = 128;

// One CTA per token and key/value head, any sizes, either activation type; one key per thread for the scores, one output
// column per thread for the weighted values.  The route of the f32 type and of head sizes beyond the tensor-core
// kernels.
template <typename T>
__global__ void __launch_bounds__(kScalarThreads)
scalar_attention_kernel(const PagedAttentionArgs<T> args) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float shared[];
    __shared__ int64_t key_rows[kScalarThreads];
    const StackAttentionShape& shape = args.shape;
    const uint32_t group = shape.heads / shape.kv_heads;
    float* query = shared;                                       // [group][dim], times scale
    float* weight = query + group * shape.dim;                   // [group][128]
    float* sum = weight + group * kScalarThreads;                // [group][vdim]
    float* top = sum + group * shape.vdim;                       // [group] running maximum
    float* denominator = top + group;                            // [group]
    float* rescale = denominator + group;                        // [group] of the current key tile
    const size_t token = blockIdx.x / shape.kv_heads;
    const uint32_t kv_head = static_cast<uint32_t>(blockIdx.x % shape.kv_heads);
    const size_t table = args.request_slots[token];
    if (table >= args.block_table_rows) {
        return;
    }
    const uint32_t position = args.positions[token];
    const uint32_t first = first_visible(position, shape.chunk);
    const T* query_row = args.query + (token * shape.heads + static_cast<size_t>(kv_head) * group) * shape.dim;
    for (uint32_t i = threadIdx.x; i < group * shape.dim; i += kScalarThreads) {
        query[i] = to_float<T>(query_row[i]) * shape.scale;
    }
    for (uint32_t i = threadIdx.x; i < group * shape.vdim; i += kScalarThreads) sum[i] = 0.0f;
    for (uint32_t i = threadIdx.x; i < group; i += kScalarThreads) {
        top[i] = -INFINITY;
        denominator[i] = 0.0f;
    }
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    for (uint32_t base = first; base <= position; base += kScalarThreads) {
        __syncthreads();
        const uint32_t key = base + threadIdx.x;
        const int64_t row = key <= position ? cache_row(args, table, key, kv_head) : -1;
        key_rows[threadIdx.x] = row;
        for (uint32_t head = 0; head < group; head += 4) {
            float dot[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            const uint32_t count = group - head < 4 ? group - head : 4;
            if (row >= 0) {
                const T* key_row = args.key_cache + row * shape.dim;
                for (uint32_t d = 0; d < shape.dim; ++d) {
                    const float value = to_float<T>(key_row[d]);
                    for (uint32_t h = 0; h < 4; ++h) {
                        if (h < count) dot[h] = fmaf(value, query[(head + h) * shape.dim + d], dot[h]);
                    }
                }
            }
            for (uint32_t h = 0; h < count; ++h) {
                weight[(head + h) * kScalarThreads + threadIdx.x] = row >= 0 ? dot[h] : -INFINITY;
            }
        }
        __syncthreads();
        for (uint32_t head = warp; head < group; head += kScalarThreads / 32) {
            float* scores = weight + head * kScalarThreads;
            float best = -INFINITY;
            for (uint32_t i = lane; i < kScalarThreads; i += 32) best = fmaxf(best, scores[i]);
            for (uint32_t delta = 16; delta > 0; delta >>= 1) {
                best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, delta));
            }
            const float before = top[head];
            const float now = fmaxf(before, best);
            float total = 0.0f;
            for (uint32_t i = lane; i < kScalarThreads; i += 32) {
                const float value = now == -INFINITY ? 0.0f : expf(scores[i] - now);
                scores[i] = value;
                total += value;
            }
            total = warp_sum(total);
            if (lane == 0) {
                const float factor = now == -INFINITY ? 1.0f : expf(before - now);
                rescale[head] = factor;
                denominator[head] = denominator[head] * factor + total;
                top[head] = now;
            }
        }
        __syncthreads();
        const uint32_t keys = position - base + 1 < kScalarThreads ? position - base + 1 : kScalarThreads;
        for (uint32_t item = threadIdx.x; item < group * shape.vdim; item += kScalarThreads) {
            const uint32_t head = item / shape.vdim;
            const uint32_t column = item % shape.vdim;
            const float* weights = weight + head * kScalarThreads;
            float value = sum[item] * rescale[head];
            for (uint32_t i = 0; i < keys; ++i) {
                if (key_rows[i] >= 0) {
                    value = fmaf(weights[i], to_float<T>(args.value_cache[key_rows[i] * shape.vdim + column]), value);
                }
            }
            sum[item] = value;
        }
    }
    __syncthreads();
    T* out = args.out + token * args.out_pitch + static_cast<size_t>(kv_head) * group * shape.vdim;
    for (uint32_t item = threadIdx.x; item < group * shape.vdim; item += kScalarThreads) {
        const float total = denominator[item / shape.vdim];
        out[item] = from_float<T>(total > 0.0f ? sum[item] / total : 0.0f);
    }
}

template <typename T>
cudaError_t launch_scalar(cudaStream_t stream, const StackAttentionLaunch& launch, size_t first_token, size_t tokens) {
    PagedAttentionArgs<T> args = paged_attention_args<T>(launch);
    args.query += first_token * launch.shape.heads * launch.shape.dim;
    args.request_slots += first_token;
    args.positions += first_token;
    args.out += first_token * launch.out_pitch;
    const size_t group = launch.shape.heads / launch.shape.kv_heads;
    const size_t shared = group * (launch.shape.dim + kScalarThreads + launch.shape.vdim + 3) * sizeof(float);
    if (shared > 227 * 1024 - 2048) {
        return cudaErrorInvalidValue;
    }
    if (shared > 40 * 1024) {
        const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(scalar_attention_kernel<T>),
                                                        cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                        static_cast<int>(shared));
        if (status != cudaSuccess) return status;
    }
    return launch_kernel(scalar_attention_kernel<T>, static_cast<unsigned int>(tokens * launch.shape.kv_heads),
                         kScalarThreads, shared, stream, 1, args);
}

}  // namespace

cudaError_t launch_projection_norm_rope(cudaStream_t stream, const ProjectionNormRopeLaunch& launch) {
    return launch.type == Activation::kF32 ? launch_post<float>(stream, launch)
                                           : launch_post<__nv_bfloat16>(stream, launch);
}

cudaError_t launch_stack_attention(cudaStream_t stream, const StackAttentionLaunch& launch) {
    const size_t tokens = launch.segments.num_tokens;
    if (launch.type == Activation::kF32) {
        return launch_scalar<float>(stream, launch, 0, tokens);
    }
    const bool scalar = option(kOptStackAttention) != 0;
    if (launch.decode_tokens > 0) {
        const cudaError_t status = !scalar && stack_attention_decode_supports(launch)
                                       ? launch_stack_attention_decode(stream, launch)
                                       : launch_scalar<__nv_bfloat16>(stream, launch, 0, launch.decode_tokens);
        if (status != cudaSuccess) return status;
    }
    if (launch.decode_tokens == tokens) {
        return cudaSuccess;
    }
    if (!scalar && stack_attention_umma_supports(launch)) {
        // segment offsets are absolute token indices, so the remaining segments are simply a later start
        StackAttentionLaunch prompts = launch;
        prompts.segments.offsets += launch.decode_tokens;
        prompts.segments.slots += launch.decode_tokens;
        prompts.segments.num_segments -= launch.decode_tokens;
        return launch_stack_attention_umma(stream, prompts);
    }
    return launch_scalar<__nv_bfloat16>(stream, launch, launch.decode_tokens, tokens - launch.decode_tokens);
}

}  // namespace lfm25
