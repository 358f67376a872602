// Shared by the attention kernels of the layer stack: their argument block and the addressing of the paged cache.
#pragma once

#include <cuda.h>

#include "common.cuh"
#include "stack_kernels.h"

namespace lfm25 {

template <typename T>
struct PagedAttentionArgs {
    StackAttentionShape shape;
    const T* query;                // [T, heads * dim]
    const T* key_cache;            // [pages, kv_heads, 16, dim]
    const T* value_cache;          // [pages, kv_heads, 16, vdim]
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* request_slots;
    const uint32_t* positions;
    StackSegments segments;
    T* out;
    size_t out_pitch;
};

template <typename T>
PagedAttentionArgs<T> paged_attention_args(const StackAttentionLaunch& launch) {
    PagedAttentionArgs<T> args;
    args.shape = launch.shape;
    args.query = static_cast<const T*>(launch.query);
    args.key_cache = static_cast<const T*>(launch.key_cache);
    args.value_cache = static_cast<const T*>(launch.value_cache);
    args.block_tables = launch.block_tables;
    args.block_table_stride = launch.block_table_stride;
    args.block_table_rows = launch.block_table_rows;
    args.num_pages = launch.num_pages;
    args.request_slots = launch.request_slots;
    args.positions = launch.positions;
    args.segments = launch.segments;
    args.out = static_cast<T*>(launch.out);
    args.out_pitch = launch.out_pitch;
    return args;
}

// First key position that `position` sees: the start of its chunk, counted from position 0 of the sequence.
__device__ __forceinline__ uint32_t first_visible(uint32_t position, uint32_t chunk) {
    return chunk == 0 ? 0u : position - position % chunk;
}

// Row of the cache (in units of one head's key or value vector) that holds key `position` of the sequence in block
// table row `table`; -1 when no page is assigned.
template <typename T>
__device__ __forceinline__ int64_t cache_row(const PagedAttentionArgs<T>& args, size_t table, uint32_t position,
                                             uint32_t kv_head) {
    const size_t index = position / kPageSize;
    if (index >= args.block_table_stride) {
        return -1;
    }
    const size_t page = args.block_tables[table * args.block_table_stride + index];
    if (page >= args.num_pages) {
        return -1;
    }
    return static_cast<int64_t>((page * args.shape.kv_heads + kv_head) * kPageSize + position % kPageSize);
}

// Tensor map of the key (value) cache: rows of one head's vector, boxes of 64 dimensions x one page, 128-byte swizzle;
// dimensions beyond the head's size read as zero.
bool make_page_map(CUtensorMap* map, const StackAttentionLaunch& launch, bool value);
// what both tensor-core kernels need of a launch: bf16, 16-byte rows, a positive scale
bool paged_copies_possible(const StackAttentionLaunch& launch);

bool stack_attention_umma_supports(const StackAttentionLaunch& launch);
cudaError_t launch_stack_attention_umma(cudaStream_t stream, const StackAttentionLaunch& launch);

// The first decode_tokens tokens (every one a segment of its own).
uint32_t stack_attention_splits(const StackAttentionShape& shape, size_t tokens, size_t context);
bool stack_attention_decode_supports(const StackAttentionLaunch& launch);
cudaError_t launch_stack_attention_decode(cudaStream_t stream, const StackAttentionLaunch& launch);

}  // namespace lfm25
