// Latent attention of the layer stack for any sizes: the norms of the two latents with the paged append, rotation of the
// queries, the plain attention kernel over cached latents, and the copy of cached contexts into contiguous rows.
#include <math.h>

#include "launch.h"
#include "options.h"
#include "stack_latent.h"

namespace lfm25 {

namespace {

constexpr uint32_t kThreads = 256;

template <typename T>
struct ProjectionArgs {
    const T* projected;
    size_t pitch;
    uint32_t q_rank, kv_rank, rot_dim, rot_dims;
    size_t latent_column;
    bool append;
    const __nv_bfloat16* query_norm;
    const __nv_bfloat16* latent_norm;
    const float* inv_freq;
    const uint32_t* positions;
    const int64_t* physical_slots;
    T* query_out;
    T* latent_cache;
    T* key_cache;
    size_t num_pages;
    float eps;
};

// One CTA per token: both latents at once, the sums of squares first.
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
latent_projection_kernel(const ProjectionArgs<T> args) {
    pdl_launch_dependents();
    __shared__ float scratch[2][kThreads / 32];
    pdl_wait();
    const size_t token = blockIdx.x;
    const T* query = args.projected + token * args.pitch;
    const T* latent = query + args.latent_column;
    float query_sum = 0.0f, latent_sum = 0.0f;
    for (uint32_t column = threadIdx.x * VEC; column < args.q_rank; column += kThreads * VEC) {
        float value[VEC];
        load_values<VEC>(query + column, value);
#pragma unroll
        for (int i = 0; i < VEC; ++i) query_sum = fmaf(value[i], value[i], query_sum);
    }
    if (args.append) {
        for (uint32_t column = threadIdx.x * VEC; column < args.kv_rank; column += kThreads * VEC) {
            float value[VEC];
            load_values<VEC>(latent + column, value);
#pragma unroll
            for (int i = 0; i < VEC; ++i) latent_sum = fmaf(value[i], value[i], latent_sum);
        }
    }
    query_sum = warp_sum(query_sum);
    latent_sum = warp_sum(latent_sum);
    const uint32_t lane = threadIdx.x & 31;
    if (lane == 0) {
        scratch[0][threadIdx.x >> 5] = query_sum;
        scratch[1][threadIdx.x >> 5] = latent_sum;
    }
    __syncthreads();
    query_sum = warp_sum(lane < kThreads / 32 ? scratch[0][lane] : 0.0f);
    latent_sum = warp_sum(lane < kThreads / 32 ? scratch[1][lane] : 0.0f);
    auto normed = [](const T* source, const __nv_bfloat16* norm, T* target, uint32_t count, float scale) {
        for (uint32_t column = threadIdx.x * VEC; column < count; column += kThreads * VEC) {
            float value[VEC], weight[VEC];
            load_values<VEC>(source + column, value);
            load_values<VEC>(norm + column, weight);
#pragma unroll
            for (int i = 0; i < VEC; ++i) value[i] *= scale * weight[i];
            store_values<VEC>(target + column, value);
        }
    };
    normed(query, args.query_norm, args.query_out + token * args.q_rank, args.q_rank,
           inverse_rms(query_sum, args.q_rank, args.eps));
    const int64_t slot = args.append ? args.physical_slots[token] : -1;
    const size_t page = slot < 0 ? args.num_pages : static_cast<size_t>(slot) / kPageSize;
    if (page >= args.num_pages) {
        return;
    }
    normed(latent, args.latent_norm, args.latent_cache + static_cast<size_t>(slot) * args.kv_rank, args.kv_rank,
           inverse_rms(latent_sum, args.kv_rank, args.eps));
    const T* key = latent + args.kv_rank;
    T* key_out = args.key_cache + static_cast<size_t>(slot) * args.rot_dim;
    const float position = static_cast<float>(args.positions[token]);
    const uint32_t half = args.rot_dims / 2;
    for (uint32_t i = threadIdx.x; i < half; i += kThreads) {
        float sine, cosine;
        sincosf(position * args.inv_freq[i], &sine, &cosine);
        const float u = to_float<T>(key[i]), v = to_float<T>(key[i + half]);
        key_out[i] = from_float<T>(u * cosine - v * sine);
        key_out[i + half] = from_float<T>(v * cosine + u * sine);
    }
    for (uint32_t i = args.rot_dims + threadIdx.x; i < args.rot_dim; i += kThreads) key_out[i] = key[i];
}

template <typename T>
cudaError_t launch_projection(cudaStream_t stream, const LatentProjectionLaunch& launch) {
    ProjectionArgs<T> args;
    args.projected = static_cast<const T*>(launch.projected);
    args.pitch = launch.pitch;
    args.q_rank = launch.q_rank;
    args.kv_rank = launch.kv_rank;
    args.rot_dim = launch.rot_dim;
    args.rot_dims = launch.rot_dims;
    args.latent_column = launch.latent_column;
    args.append = launch.append;
    args.query_norm = static_cast<const __nv_bfloat16*>(launch.query_norm);
    args.latent_norm = static_cast<const __nv_bfloat16*>(launch.latent_norm);
    args.inv_freq = launch.inv_freq;
    args.positions = launch.positions;
    args.physical_slots = launch.physical_slots;
    args.query_out = static_cast<T*>(launch.query_out);
    args.latent_cache = static_cast<T*>(launch.latent_cache);
    args.key_cache = static_cast<T*>(launch.key_cache);
    args.num_pages = launch.num_pages;
    args.eps = launch.eps;
    const bool vector = launch.q_rank % 8 == 0 && launch.kv_rank % 8 == 0 && launch.latent_column % 8 == 0 &&
                        launch.pitch % 8 == 0 && aligned_to(launch.projected, 16) && aligned_to(launch.query_norm, 16) &&
                        aligned_to(launch.latent_norm, 16) && aligned_to(launch.query_out, 16) &&
                        aligned_to(launch.latent_cache, 16);
    return launch_kernel(vector ? latent_projection_kernel<T, 8> : latent_projection_kernel<T, 1>,
                         static_cast<unsigned int>(launch.num_tokens), kThreads, 0, stream, 1, args);
}

// One CTA per token: the angles once, then every head's pairs.
template <typename T>
__global__ void __launch_bounds__(kThreads)
rotate_queries_kernel(T* __restrict__ query, size_t token_pitch, const float* __restrict__ inv_freq,
                      const uint32_t* __restrict__ positions, uint32_t heads, uint32_t dim, uint32_t rot_dim,
                      uint32_t half) {
    pdl_launch_dependents();
    extern __shared__ float2 angles[];                // [half] (cos, sin)
    pdl_wait();
    const float position = static_cast<float>(positions[blockIdx.x]);
    for (uint32_t i = threadIdx.x; i < half; i += kThreads) {
        float sine, cosine;
        sincosf(position * inv_freq[i], &sine, &cosine);
        angles[i] = make_float2(cosine, sine);
    }
    __syncthreads();
    const size_t pitch = dim + rot_dim;
    T* rows = query + blockIdx.x * token_pitch + dim;
    for (uint32_t item = threadIdx.x; item < heads * half; item += kThreads) {
        const uint32_t i = item % half;
        T* pair = rows + item / half * pitch + i;
        const float2 angle = angles[i];
        const float u = to_float<T>(pair[0]), v = to_float<T>(pair[half]);
        pair[0] = from_float<T>(u * angle.x - v * angle.y);
        pair[half] = from_float<T>(v * angle.x + u * angle.y);
    }
}

// ------------------------------------------------------------------------------------------------ plain attention

constexpr uint32_t kPlainThreads = 128;
constexpr uint32_t kPlainHeads = 4;

// One CTA per token and up to four heads, any sizes, either activation type; one key per thread for the scores, one latent
// column per thread for the weighted sum.  The route of the f32 type and of sizes beyond the tensor-core kernel.
template <typename T>
__global__ void __launch_bounds__(kPlainThreads)
latent_attention_plain_kernel(const LatentArgs<T> args, uint32_t head_blocks) {
    pdl_launch_dependents();
    extern __shared__ float shared[];
    __shared__ int64_t key_rows[kPlainThreads];
    __shared__ float top[kPlainHeads], denominator[kPlainHeads], rescale[kPlainHeads];
    const LatentAttentionShape& shape = args.shape;
    float* latent_query = shared;                                     // [heads][kv_rank], times scale
    float* rotated_query = latent_query + kPlainHeads * shape.kv_rank;
    float* weight = rotated_query + kPlainHeads * shape.rot_dim;      // [heads][128]
    float* sum = weight + kPlainHeads * kPlainThreads;                // [heads][kv_rank]
    pdl_wait();
    const size_t token = blockIdx.x / head_blocks;
    const uint32_t head0 = static_cast<uint32_t>(blockIdx.x % head_blocks) * kPlainHeads;
    const uint32_t count = shape.heads - head0 < kPlainHeads ? shape.heads - head0 : kPlainHeads;
    const size_t table = args.request_slots[token];
    if (table >= args.block_table_rows) {
        return;
    }
    const uint32_t position = args.positions[token];
    const size_t query_head = shape.dim + shape.rot_dim;
    for (uint32_t i = threadIdx.x; i < kPlainHeads * shape.kv_rank; i += kPlainThreads) {
        const uint32_t head = i / shape.kv_rank;
        latent_query[i] =
            head < count ? to_float<T>(args.absorbed[(token * shape.heads + head0) * shape.kv_rank + i]) * shape.scale
                         : 0.0f;
        sum[i] = 0.0f;
    }
    for (uint32_t i = threadIdx.x; i < kPlainHeads * shape.rot_dim; i += kPlainThreads) {
        const uint32_t head = i / shape.rot_dim;
        rotated_query[i] =
            head < count ? to_float<T>(args.query[token * args.query_pitch + (head0 + head) * query_head + shape.dim +
                                                  i % shape.rot_dim]) * shape.scale
                         : 0.0f;
    }
    if (threadIdx.x < kPlainHeads) {
        top[threadIdx.x] = -INFINITY;
        denominator[threadIdx.x] = 0.0f;
    }
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    for (uint32_t base = 0; base <= position; base += kPlainThreads) {
        __syncthreads();
        const uint32_t key = base + threadIdx.x;
        const int64_t row = key <= position ? latent_row(args, table, key) : -1;
        key_rows[threadIdx.x] = row;
        float dot[kPlainHeads] = {};
        if (row >= 0) {
            const T* latent = args.latent_cache + row * shape.kv_rank;
            for (uint32_t d = 0; d < shape.kv_rank; ++d) {
                const float value = to_float<T>(latent[d]);
#pragma unroll
                for (uint32_t h = 0; h < kPlainHeads; ++h) {
                    dot[h] = fmaf(value, latent_query[h * shape.kv_rank + d], dot[h]);
                }
            }
            const T* rotated = args.key_cache + row * shape.rot_dim;
            for (uint32_t d = 0; d < shape.rot_dim; ++d) {
                const float value = to_float<T>(rotated[d]);
#pragma unroll
                for (uint32_t h = 0; h < kPlainHeads; ++h) {
                    dot[h] = fmaf(value, rotated_query[h * shape.rot_dim + d], dot[h]);
                }
            }
        }
#pragma unroll
        for (uint32_t h = 0; h < kPlainHeads; ++h) {
            weight[h * kPlainThreads + threadIdx.x] = row >= 0 ? dot[h] : -INFINITY;
        }
        __syncthreads();
        if (warp < kPlainHeads) {
            float* scores = weight + warp * kPlainThreads;
            float best = -INFINITY;
            for (uint32_t i = lane; i < kPlainThreads; i += 32) best = fmaxf(best, scores[i]);
            for (uint32_t delta = 16; delta > 0; delta >>= 1) {
                best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, delta));
            }
            const float before = top[warp];
            const float now = fmaxf(before, best);
            float total = 0.0f;
            for (uint32_t i = lane; i < kPlainThreads; i += 32) {
                const float value = now == -INFINITY ? 0.0f : expf(scores[i] - now);
                scores[i] = value;
                total += value;
            }
            total = warp_sum(total);
            __syncwarp();
            if (lane == 0) {
                const float factor = now == -INFINITY ? 1.0f : expf(before - now);
                rescale[warp] = factor;
                denominator[warp] = denominator[warp] * factor + total;
                top[warp] = now;
            }
        }
        __syncthreads();
        const uint32_t keys = position - base + 1 < kPlainThreads ? position - base + 1 : kPlainThreads;
        for (uint32_t column = threadIdx.x; column < shape.kv_rank; column += kPlainThreads) {
            float value[kPlainHeads];
#pragma unroll
            for (uint32_t h = 0; h < kPlainHeads; ++h) value[h] = sum[h * shape.kv_rank + column] * rescale[h];
            for (uint32_t i = 0; i < keys; ++i) {
                if (key_rows[i] >= 0) {
                    const float entry = to_float<T>(args.latent_cache[key_rows[i] * shape.kv_rank + column]);
#pragma unroll
                    for (uint32_t h = 0; h < kPlainHeads; ++h) {
                        value[h] = fmaf(weight[h * kPlainThreads + i], entry, value[h]);
                    }
                }
            }
#pragma unroll
            for (uint32_t h = 0; h < kPlainHeads; ++h) sum[h * shape.kv_rank + column] = value[h];
        }
    }
    __syncthreads();
    T* out = args.out + (token * shape.heads + head0) * shape.kv_rank;
    for (uint32_t i = threadIdx.x; i < count * shape.kv_rank; i += kPlainThreads) {
        const float total = denominator[i / shape.kv_rank];
        out[i] = from_float<T>(total > 0.0f ? sum[i] / total : 0.0f);
    }
}

template <typename T>
cudaError_t launch_plain(cudaStream_t stream, const LatentAttentionLaunch& launch) {
    const LatentArgs<T> args = latent_args<T>(launch);
    const uint32_t head_blocks = (launch.shape.heads + kPlainHeads - 1) / kPlainHeads;
    const size_t shared =
        kPlainHeads * (2 * static_cast<size_t>(launch.shape.kv_rank) + launch.shape.rot_dim + kPlainThreads) * sizeof(float);
    if (shared > 200 * 1024) {
        return cudaErrorInvalidValue;
    }
    if (shared > 40 * 1024) {
        const cudaError_t status =
            cudaFuncSetAttribute(reinterpret_cast<const void*>(latent_attention_plain_kernel<T>),
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
        if (status != cudaSuccess) return status;
    }
    return launch_kernel(latent_attention_plain_kernel<T>, static_cast<unsigned int>(launch.tokens * head_blocks),
                         kPlainThreads, shared, stream, 1, args, head_blocks);
}

// ------------------------------------------------------------------------------------------------ contiguous contexts

// One warp; segments in rounds of 32.
__global__ void context_bases_kernel(const StackSegments segments, const uint32_t* __restrict__ positions,
                                     uint32_t first_segment, uint32_t* __restrict__ bases) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t lane = threadIdx.x;
    uint32_t before = 0;
    for (uint32_t round = 0; round < segments.num_segments; round += 32) {
        const uint32_t segment = round + lane;
        uint32_t rows = 0;
        if (segment >= first_segment && segment < segments.num_segments) {
            const uint32_t begin = segments.offsets[segment], end = segments.offsets[segment + 1];
            if (end > begin && end <= segments.num_tokens) {
                rows = (positions[end - 1] + kContextRows) / kContextRows * kContextRows;
            }
        }
        uint32_t inclusive = rows;
#pragma unroll
        for (uint32_t delta = 1; delta < 32; delta <<= 1) {
            const uint32_t other = __shfl_up_sync(0xffffffffu, inclusive, delta);
            inclusive += lane >= delta ? other : 0u;
        }
        if (segment < segments.num_segments) bases[segment] = before + inclusive - rows;
        before += __shfl_sync(0xffffffffu, inclusive, 31);
    }
    if (lane == 0) bases[segments.num_segments] = before;
}

template <typename T>
struct GatherArgs {
    StackSegments segments;
    uint32_t first_segment;
    const uint32_t* bases;
    const uint32_t* positions;
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    uint32_t kv_rank, rot_dim;
    const T* latent_cache;
    const T* key_cache;
    T* latents;
    T* keys;
    size_t rows;
};

// One CTA per 16 rows (one page; contexts start at multiples of 64)
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
gather_context_kernel(const GatherArgs<T> args) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t row0 = blockIdx.x * kPageSize;
    uint32_t low = args.first_segment, high = static_cast<uint32_t>(args.segments.num_segments);
    while (low + 1 < high) {                        // the last segment that starts at or before row0
        const uint32_t middle = (low + high) / 2;
        if (args.bases[middle] <= row0) {
            low = middle;
        } else {
            high = middle;
        }
    }
    const uint32_t context = args.positions[args.segments.offsets[low + 1] - 1] + 1;
    const uint32_t key0 = row0 - args.bases[low];
    const size_t table = args.segments.slots[low];
    size_t page = args.num_pages;
    if (key0 < context && table < args.block_table_rows && key0 / kPageSize < args.block_table_stride) {
        page = args.block_tables[table * args.block_table_stride + key0 / kPageSize];
    }
    const uint32_t valid = page < args.num_pages ? (context - key0 < kPageSize ? context - key0 : kPageSize) : 0;
    auto copy = [&](const T* source, T* target, uint32_t width) {
        for (uint32_t at = threadIdx.x * VEC; at < kPageSize * width; at += kThreads * VEC) {
            float value[VEC];
            if (at < valid * width) {
                load_values<VEC>(source + page * kPageSize * width + at, value);
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) value[i] = 0.0f;
            }
            store_values<VEC>(target + static_cast<size_t>(row0) * width + at, value);
        }
    };
    copy(args.latent_cache, args.latents, args.kv_rank);
    copy(args.key_cache, args.keys, args.rot_dim);
}

template <typename T>
cudaError_t launch_gather(cudaStream_t stream, const GatherContextLaunch& launch) {
    GatherArgs<T> args;
    args.segments = launch.segments;
    args.first_segment = static_cast<uint32_t>(launch.first_segment);
    args.bases = launch.bases;
    args.positions = launch.positions;
    args.block_tables = launch.block_tables;
    args.block_table_stride = launch.block_table_stride;
    args.block_table_rows = launch.block_table_rows;
    args.num_pages = launch.num_pages;
    args.kv_rank = launch.kv_rank;
    args.rot_dim = launch.rot_dim;
    args.latent_cache = static_cast<const T*>(launch.latent_cache);
    args.key_cache = static_cast<const T*>(launch.key_cache);
    args.latents = static_cast<T*>(launch.latents);
    args.keys = static_cast<T*>(launch.keys);
    args.rows = launch.rows;
    const bool vector = launch.kv_rank % 8 == 0 && launch.rot_dim % 8 == 0 && aligned_to(launch.latent_cache, 16) &&
                        aligned_to(launch.key_cache, 16) && aligned_to(launch.latents, 16) && aligned_to(launch.keys, 16);
    return launch_kernel(vector ? gather_context_kernel<T, 8> : gather_context_kernel<T, 1>,
                         static_cast<unsigned int>(launch.rows / kPageSize), kThreads, 0, stream, 1, args);
}

}  // namespace

cudaError_t launch_latent_projection(cudaStream_t stream, const LatentProjectionLaunch& launch) {
    return launch.type == Activation::kF32 ? launch_projection<float>(stream, launch)
                                           : launch_projection<__nv_bfloat16>(stream, launch);
}

cudaError_t launch_rotate_queries(cudaStream_t stream, Activation type, void* query, size_t pitch, const float* inv_freq,
                                  const uint32_t* positions, size_t tokens, uint32_t heads, uint32_t dim,
                                  uint32_t rot_dim, uint32_t rot_dims) {
    if (rot_dims == 0) {
        return cudaSuccess;
    }
    const uint32_t half = rot_dims / 2;
    auto go = [&](auto* typed) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(rotate_queries_kernel<T>, static_cast<unsigned int>(tokens), kThreads, half * sizeof(float2),
                             stream, 1, static_cast<T*>(query), pitch, inv_freq, positions, heads, dim, rot_dim, half);
    };
    return type == Activation::kF32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

cudaError_t launch_latent_attention(cudaStream_t stream, const LatentAttentionLaunch& launch) {
    if (launch.type == Activation::kF32) {
        return launch_plain<float>(stream, launch);
    }
    if (option(kOptStackAttention) == 0 && latent_attention_umma_supports(launch)) {
        return launch_latent_attention_umma(stream, launch);
    }
    return launch_plain<__nv_bfloat16>(stream, launch);
}

cudaError_t launch_context_bases(cudaStream_t stream, const StackSegments& segments, const uint32_t* positions,
                                 size_t first_segment, uint32_t* bases) {
    return launch_kernel(context_bases_kernel, 1, 32, 0, stream, 1, segments, positions,
                         static_cast<uint32_t>(first_segment), bases);
}

cudaError_t launch_gather_context(cudaStream_t stream, const GatherContextLaunch& launch) {
    return launch.type == Activation::kF32 ? launch_gather<float>(stream, launch)
                                           : launch_gather<__nv_bfloat16>(stream, launch);
}

}  // namespace lfm25
