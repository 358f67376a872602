// Device helpers of the layer-stack kernels: typed loads and stores of 1 or 8 consecutive activations, reductions,
// and the mapping of CTAs onto row tiles that never cross a segment border.
#pragma once

#include "common.cuh"
#include "stack_kernels.h"

namespace lfm25 {

template <typename T>
__device__ __forceinline__ float to_float(T value);
template <>
__device__ __forceinline__ float to_float<float>(float value) {
    return value;
}
template <>
__device__ __forceinline__ float to_float<__nv_bfloat16>(__nv_bfloat16 value) {
    return __bfloat162float(value);
}
template <typename T>
__device__ __forceinline__ T from_float(float value);
template <>
__device__ __forceinline__ float from_float<float>(float value) {
    return value;
}
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float value) {
    return __float2bfloat16_rn(value);
}

// VEC consecutive values (1, or 8 with 16-byte aligned bf16 / 32-byte aligned f32)
template <int VEC>
__device__ __forceinline__ void load_values(const __nv_bfloat16* source, float (&out)[VEC]) {
    if constexpr (VEC == 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(source);
        const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int pair = 0; pair < 4; ++pair) {
            const float2 both = __bfloat1622float2(pairs[pair]);
            out[2 * pair] = both.x;
            out[2 * pair + 1] = both.y;
        }
    } else {
        static_assert(VEC == 1, "1 or 8 values");
        out[0] = __bfloat162float(*source);
    }
}
template <int VEC>
__device__ __forceinline__ void load_values(const float* source, float (&out)[VEC]) {
    if constexpr (VEC == 8) {
        const float4 low = reinterpret_cast<const float4*>(source)[0];
        const float4 high = reinterpret_cast<const float4*>(source)[1];
        out[0] = low.x; out[1] = low.y; out[2] = low.z; out[3] = low.w;
        out[4] = high.x; out[5] = high.y; out[6] = high.z; out[7] = high.w;
    } else {
        out[0] = *source;
    }
}
template <int VEC>
__device__ __forceinline__ void store_values(__nv_bfloat16* target, const float (&values)[VEC]) {
    if constexpr (VEC == 8) {
        uint4 raw;
        raw.x = pack_bf16x2(values[0], values[1]);
        raw.y = pack_bf16x2(values[2], values[3]);
        raw.z = pack_bf16x2(values[4], values[5]);
        raw.w = pack_bf16x2(values[6], values[7]);
        *reinterpret_cast<uint4*>(target) = raw;
    } else {
        *target = __float2bfloat16_rn(values[0]);
    }
}
template <int VEC>
__device__ __forceinline__ void store_values(float* target, const float (&values)[VEC]) {
    if constexpr (VEC == 8) {
        reinterpret_cast<float4*>(target)[0] = make_float4(values[0], values[1], values[2], values[3]);
        reinterpret_cast<float4*>(target)[1] = make_float4(values[4], values[5], values[6], values[7]);
    } else {
        *target = values[0];
    }
}

// 16 bytes global -> shared behind the thread's back; `inside` false: zeros (the source is not read)
__device__ __forceinline__ void copy_async_16(void* target, const void* source, bool inside) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(target)), "l"(source), "r"(inside ? 16 : 0)
                 : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <uint32_t NEWER>
__device__ __forceinline__ void copy_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(NEWER) : "memory");
}

__device__ __forceinline__ float warp_sum(float value) {
#pragma unroll
    for (uint32_t delta = 16; delta > 0; delta >>= 1) {
        value += __shfl_xor_sync(0xffffffffu, value, delta);
    }
    return value;
}

// Sum over the CTA; every thread gets it.  `scratch` holds one float per warp and is free again after the call's
// second barrier, so consecutive calls may share it.
__device__ __forceinline__ float block_sum(float value, float* scratch) {
    value = warp_sum(value);
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    if (lane == 0) {
        scratch[warp] = value;
    }
    __syncthreads();
    const float total = warp_sum(lane < (blockDim.x >> 5) ? scratch[lane] : 0.0f);
    __syncthreads();
    return total;
}

// x / sqrt(mean + eps) uses this factor everywhere, with both operations correctly rounded
__device__ __forceinline__ float inverse_rms(float sum_of_squares, size_t count, float eps) {
    return 1.0f / sqrtf(sum_of_squares / static_cast<float>(count) + eps);
}

__device__ __forceinline__ float sigmoidf(float z) { return 1.0f / (1.0f + expf(-z)); }

// The tokens that one CTA works on: `count` rows from `first`, all of segment `segment` = [begin, end).
struct SegmentTile {
    uint32_t segment;
    uint32_t begin, end;
    uint32_t first, count;   // count == 0: no work for this CTA
};

// Tile `index` of the step when every segment is cut into tiles of `rows` tokens, counted over all segments in order.
// Called by whole warps; every lane gets the same answer.
__device__ __forceinline__ SegmentTile locate_tile(const StackSegments& segments, uint32_t rows, uint32_t index) {
    SegmentTile tile = {0, 0, 0, 0, 0};
    if (segments.offsets == nullptr) {
        if (index < segments.num_tokens) {
            tile = {index, index, index + 1, index, 1};
        }
        return tile;
    }
    const uint32_t lane = threadIdx.x & 31;
    uint32_t before = 0;
    for (uint32_t base = 0; base < segments.num_segments; base += 32) {
        const uint32_t segment = base + lane;
        uint32_t begin = 0, end = 0;
        if (segment < segments.num_segments) {
            begin = segments.offsets[segment];
            end = segments.offsets[segment + 1];
            end = end < segments.num_tokens ? end : static_cast<uint32_t>(segments.num_tokens);
            end = end > begin ? end : begin;
        }
        const uint32_t tiles = (end - begin + rows - 1) / rows;
        uint32_t inclusive = tiles;
#pragma unroll
        for (uint32_t delta = 1; delta < 32; delta <<= 1) {
            const uint32_t other = __shfl_up_sync(0xffffffffu, inclusive, delta);
            inclusive += lane >= delta ? other : 0u;
        }
        const bool mine = index >= before + inclusive - tiles && index < before + inclusive;
        const uint32_t owners = __ballot_sync(0xffffffffu, mine);
        if (owners != 0) {
            const int owner = __ffs(static_cast<int>(owners)) - 1;
            const uint32_t within = index - before - (inclusive - tiles);
            const uint32_t first = begin + within * rows;
            const uint32_t count = end - first < rows ? end - first : rows;
            tile.segment = __shfl_sync(0xffffffffu, segment, owner);
            tile.begin = __shfl_sync(0xffffffffu, begin, owner);
            tile.end = __shfl_sync(0xffffffffu, end, owner);
            tile.first = __shfl_sync(0xffffffffu, first, owner);
            tile.count = __shfl_sync(0xffffffffu, count, owner);
            return tile;
        }
        before += __shfl_sync(0xffffffffu, inclusive, 31);
    }
    return tile;
}

// Upper bound of the number of tiles locate_tile() can return work for.
inline size_t tile_bound(const StackSegments& segments, size_t rows) {
    if (segments.offsets == nullptr) {
        return segments.num_tokens;
    }
    return segments.num_tokens / rows + segments.num_segments;
}

inline bool aligned_to(const void* pointer, size_t bytes) {
    return (reinterpret_cast<uintptr_t>(pointer) & (bytes - 1)) == 0;
}

}  // namespace lfm25
