// Shared by the latent-attention kernels of the layer stack: their argument block and the addressing of the paged cache.
#pragma once

#include "stack_common.cuh"

namespace lfm25 {

constexpr uint32_t kContextRows = 64;    // a context's rows in scratch are a multiple of this

template <typename T>
struct LatentArgs {
    LatentAttentionShape shape;
    const T* absorbed;             // [T, heads, kv_rank]
    const T* query;                // [T, heads, dim + rot_dim], rows query_pitch apart
    size_t query_pitch;
    const T* latent_cache;         // [pages, 16, kv_rank]
    const T* key_cache;            // [pages, 16, rot_dim]
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* request_slots;
    const uint32_t* positions;
    T* out;                        // [T, heads, kv_rank]
};

template <typename T>
LatentArgs<T> latent_args(const LatentAttentionLaunch& launch) {
    LatentArgs<T> args;
    args.shape = launch.shape;
    args.absorbed = static_cast<const T*>(launch.absorbed);
    args.query = static_cast<const T*>(launch.query);
    args.query_pitch = launch.query_pitch;
    args.latent_cache = static_cast<const T*>(launch.latent_cache);
    args.key_cache = static_cast<const T*>(launch.key_cache);
    args.block_tables = launch.block_tables;
    args.block_table_stride = launch.block_table_stride;
    args.block_table_rows = launch.block_table_rows;
    args.num_pages = launch.num_pages;
    args.request_slots = launch.request_slots;
    args.positions = launch.positions;
    args.out = static_cast<T*>(launch.out);
    return args;
}

// Cache row of key `position` of the sequence in block table row `table`; -1 when no page is assigned.
template <typename T>
__device__ __forceinline__ int64_t latent_row(const LatentArgs<T>& args, size_t table, uint32_t position) {
    const size_t index = position / kPageSize;
    if (index >= args.block_table_stride) {
        return -1;
    }
    const size_t page = args.block_tables[table * args.block_table_stride + index];
    return page < args.num_pages ? static_cast<int64_t>(page * kPageSize + position % kPageSize) : -1;
}

uint32_t latent_attention_splits(size_t clusters, size_t context, uint32_t latent_chunks);
bool latent_attention_umma_supports(const LatentAttentionLaunch& launch);
cudaError_t launch_latent_attention_umma(cudaStream_t stream, const LatentAttentionLaunch& launch);

}  // namespace lfm25
