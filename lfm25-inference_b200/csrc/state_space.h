// Shared by the kernels of the state-space recurrence: their argument block and what a token contributes to a head.
#pragma once

#include "stack_common.cuh"

namespace lfm25 {

template <typename T>
struct StateSpaceArgs {
    StackSegments segments;
    uint32_t heads, groups, size, vdim;
    const T* mixed;                // x [heads, vdim] | B [groups, size] | C [groups, size]
    size_t mixed_pitch;
    const T* raw_step;
    size_t step_pitch;
    const __nv_bfloat16* step_bias;
    const __nv_bfloat16* log_rate;
    const __nv_bfloat16* skip;
    StackRecord record;
    T* out;                        // [T, heads * vdim]
};

template <typename T>
StateSpaceArgs<T> state_space_args(const StateSpaceLaunch& launch) {
    StateSpaceArgs<T> args;
    args.segments = launch.segments;
    args.heads = launch.heads;
    args.groups = launch.groups;
    args.size = launch.size;
    args.vdim = launch.vdim;
    args.mixed = static_cast<const T*>(launch.mixed);
    args.mixed_pitch = launch.mixed_pitch;
    args.raw_step = static_cast<const T*>(launch.raw_step);
    args.step_pitch = launch.step_pitch;
    args.step_bias = static_cast<const __nv_bfloat16*>(launch.step_bias);
    args.log_rate = static_cast<const __nv_bfloat16*>(launch.log_rate);
    args.skip = static_cast<const __nv_bfloat16*>(launch.skip);
    args.record = launch.record;
    args.out = static_cast<T*>(launch.out);
    return args;
}

// State of one head of a request slot, [size, vdim]
template <typename T>
__device__ __forceinline__ float* state_of(const StateSpaceArgs<T>& args, size_t slot, uint32_t head) {
    float* base = reinterpret_cast<float*>(static_cast<unsigned char*>(args.record.base) + slot * args.record.stride +
                                           args.record.offset);
    return base + static_cast<size_t>(head) * args.size * args.vdim;
}

// dt = log(1 + exp(raw + bias)), without overflow
template <typename T>
__device__ __forceinline__ float step_size(const StateSpaceArgs<T>& args, size_t token, uint32_t head) {
    const float z = to_float<T>(args.raw_step[token * args.step_pitch + head]) + __bfloat162float(args.step_bias[head]);
    return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
}

// The state decays by exp(-rate dt)
template <typename T>
__device__ __forceinline__ float state_rate(const StateSpaceArgs<T>& args, uint32_t head) {
    return expf(__bfloat162float(args.log_rate[head]));
}

bool state_space_chunk_supports(const StateSpaceLaunch& launch);
cudaError_t launch_state_space_chunk(cudaStream_t stream, const StateSpaceLaunch& launch);

}  // namespace lfm25
