// State-space mixer of the layer stack: channel convolution with SiLU, the recurrence S <- a S + dt B x^T, y = S^T C as a
// decode kernel and as a token-by-token kernel for any sizes, and the gated norm behind it.
#include <math.h>

#include <algorithm>

#include "launch.h"
#include "options.h"
#include "state_space.h"

namespace lfm25 {

namespace {

// ------------------------------------------------------------------------------------------------ channel convolution

// The logistic function, to the accuracy that a result in T can show
template <typename T>
__device__ __forceinline__ float sigmoid_of(float z) {
    return sizeof(T) == 4 ? sigmoidf(z) : __fdividef(1.0f, 1.0f + __expf(-z));
}

// VEC consecutive values as they lie in memory
template <typename T, int VEC>
struct Vector {
    static constexpr int kWords = VEC * sizeof(T) >= 16 ? VEC * sizeof(T) / 16 : 1;
    uint4 words[kWords];
    T single;
    __device__ __forceinline__ void load(const T* source) {
        if constexpr (VEC == 1) {
            single = *source;
        } else {
#pragma unroll
            for (int i = 0; i < kWords; ++i) words[i] = reinterpret_cast<const uint4*>(source)[i];
        }
    }
    __device__ __forceinline__ void values(float (&out)[VEC]) const {
        if constexpr (VEC == 1) {
            out[0] = to_float<T>(single);
        } else {
            load_values<VEC>(reinterpret_cast<const T*>(words), out);
        }
    }
};

constexpr uint32_t kConvThreads = 128;
constexpr uint32_t kConvRows = 16;

template <typename T>
struct ConvArgs {
    StackSegments segments;
    const T* x;
    size_t pitch;
    const __nv_bfloat16* conv;
    const __nv_bfloat16* bias;
    uint32_t taps;
    uint32_t tile_rows;
    uint32_t channel_blocks;
    StackRecord record;
    T* out;
    size_t channels;
};

// One CTA per tile of tokens of one segment and block of channels, one thread per vector of channels.  Only the segment's
// first tile reads the record (a tile is at least as long as the history), and the same threads replace it afterwards.
// TAPS: number of taps known at compile time, whose weights and window then stay in registers; 0 = any.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kConvThreads)
channel_conv_kernel(const ConvArgs<T> args) {
    pdl_launch_dependents();
    const size_t channel =
        (static_cast<size_t>(blockIdx.x % args.channel_blocks) * kConvThreads + threadIdx.x) * VEC;
    const bool inside = channel < args.channels;
    float bias[VEC] = {}, tap[TAPS > 0 ? TAPS : 1][VEC];
    if (inside) {
        load_values<VEC>(args.bias + channel, bias);
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) load_values<VEC>(args.conv + j * args.channels + channel, tap[j]);
        }
    }
    pdl_wait();
    const SegmentTile tile = locate_tile(args.segments, args.tile_rows, blockIdx.x / args.channel_blocks);
    if (tile.count == 0 || !inside) {
        return;
    }
    const size_t slot = args.segments.slots[tile.segment];
    if (slot >= args.segments.num_request_slots) {
        return;
    }
    const int32_t history = static_cast<int32_t>(args.taps) - 1;
    T* record = reinterpret_cast<T*>(static_cast<unsigned char*>(args.record.base) + slot * args.record.stride +
                                     args.record.offset) + channel;
    const T* inputs = args.x + static_cast<size_t>(tile.begin) * args.pitch + channel;
    // the input `offset` tokens behind the segment's first one; negative offsets lie in the record
    auto load_input = [&](int32_t offset, float (&value)[VEC]) {
        if (offset < 0) {
            load_values<VEC>(record + (history + offset) * args.channels, value);
        } else {
            load_values<VEC>(inputs + offset * args.pitch, value);
        }
    };
    const int32_t first = static_cast<int32_t>(tile.first - tile.begin);
    T* out = args.out + static_cast<size_t>(tile.first) * args.channels + channel;
    if constexpr (TAPS > 0) {
        float window[TAPS][VEC];
#pragma unroll
        for (int j = 1; j < TAPS; ++j) load_input(first - (TAPS - j), window[j]);
        constexpr uint32_t kBatch = 8;               // rows whose loads are in flight together
        for (uint32_t base = 0; base < tile.count; base += kBatch) {
            Vector<T, VEC> next[kBatch];
#pragma unroll
            for (uint32_t i = 0; i < kBatch; ++i) {
                if (base + i < tile.count) next[i].load(inputs + (first + base + i) * args.pitch);
            }
#pragma unroll
            for (uint32_t step = 0; step < kBatch; ++step) {
                if (base + step >= tile.count) break;
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) {
#pragma unroll
                    for (int i = 0; i < VEC; ++i) window[j][i] = window[j + 1][i];
                }
                next[step].values(window[TAPS - 1]);
                float sum[VEC];
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    sum[i] = bias[i];
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) sum[i] = fmaf(tap[j][i], window[j][i], sum[i]);
                    sum[i] *= sigmoid_of<T>(sum[i]);
                }
                store_values<VEC>(out + (base + step) * args.channels, sum);
            }
        }
    } else {
        for (uint32_t row = 0; row < tile.count; ++row) {
            float sum[VEC], value[VEC], weight[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum[i] = bias[i];
            for (int32_t j = 0; j <= history; ++j) {
                load_input(first + static_cast<int32_t>(row) - history + j, value);
                load_values<VEC>(args.conv + j * args.channels + channel, weight);
#pragma unroll
                for (int i = 0; i < VEC; ++i) sum[i] = fmaf(weight[i], value[i], sum[i]);
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum[i] *= sigmoid_of<T>(sum[i]);
            store_values<VEC>(out + row * args.channels, sum);
        }
    }
    if (first == 0) {
        const int32_t length = static_cast<int32_t>(tile.end - tile.begin);
        for (int32_t i = 0; i < history; ++i) {      // ascending: only rows that are still to be written are read
            float value[VEC];
            load_input(length - history + i, value);
            store_values<VEC>(record + i * args.channels, value);
        }
    }
}

template <typename T>
cudaError_t launch_conv(cudaStream_t stream, const ChannelConvLaunch& launch) {
    ConvArgs<T> args;
    args.segments = launch.segments;
    args.x = static_cast<const T*>(launch.x);
    args.pitch = launch.pitch;
    args.conv = static_cast<const __nv_bfloat16*>(launch.conv);
    args.bias = static_cast<const __nv_bfloat16*>(launch.bias);
    args.taps = launch.taps;
    args.tile_rows = launch.segments.offsets == nullptr ? 1 : std::max(kConvRows, launch.taps - 1);
    args.record = launch.record;
    args.out = static_cast<T*>(launch.out);
    args.channels = launch.channels;
    const bool vector = launch.channels % 8 == 0 && launch.pitch % 8 == 0 && aligned_to(launch.x, 16) &&
                        aligned_to(launch.conv, 16) && aligned_to(launch.bias, 16) && aligned_to(launch.out, 16) &&
                        aligned_to(launch.record.base, 16) && launch.record.stride % 16 == 0 &&
                        launch.record.offset % 16 == 0;
    const size_t per_cta = static_cast<size_t>(kConvThreads) * (vector ? 8 : 1);
    args.channel_blocks = static_cast<uint32_t>((launch.channels + per_cta - 1) / per_cta);
    void (*kernel)(const ConvArgs<T>) = channel_conv_kernel<T, 1, 0>;
    if (vector) kernel = launch.taps == 4 ? channel_conv_kernel<T, 8, 4> : channel_conv_kernel<T, 8, 0>;
    return launch_kernel(kernel,
                         static_cast<unsigned int>(tile_bound(launch.segments, args.tile_rows) * args.channel_blocks),
                         kConvThreads, 0, stream, 1, args);
}

// ------------------------------------------------------------------------------------------------ decode

constexpr uint32_t kDecodeThreads = 256;

// One CTA per token and head.  A thread owns four neighbouring columns of the state in every `slices`-th row, so that the
// state streams through registers once in 16-byte pieces; the rows' contributions to y meet in shared memory.
template <typename T>
__global__ void __launch_bounds__(kDecodeThreads)
state_space_decode_kernel(const StateSpaceArgs<T> args) {
    pdl_launch_dependents();
    extern __shared__ float shared[];
    float* b = shared;                       // [size]
    float* c = b + args.size;                // [size]
    float* partial = shared + (2 * args.size + 3) / 4 * 4;   // [slices][vdim], 16-byte aligned
    pdl_wait();
    const uint32_t head = blockIdx.x % args.heads;
    const uint32_t token = blockIdx.x / args.heads;
    const size_t slot = args.segments.slots[token];
    if (slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t group = head / (args.heads / args.groups);
    const size_t inner = static_cast<size_t>(args.heads) * args.vdim;
    const T* row = args.mixed + token * args.mixed_pitch;
    const uint32_t quads = args.vdim / 4;
    const uint32_t slices = kDecodeThreads / quads;
    const uint32_t slice = threadIdx.x / quads;
    const uint32_t column = threadIdx.x % quads * 4;
    float4* state = reinterpret_cast<float4*>(state_of(args, slot, head) + column);
    constexpr uint32_t kBatch = 8;
    float4 held[kBatch];
    auto load_batch = [&](uint32_t first) {
#pragma unroll
        for (uint32_t i = 0; i < kBatch; ++i) {
            const uint32_t n = first + i * slices;
            if (slice < slices && n < args.size) held[i] = state[static_cast<size_t>(n) * quads];
        }
    };
    load_batch(slice);
    for (uint32_t n = threadIdx.x; n < args.size; n += kDecodeThreads) {
        b[n] = to_float<T>(row[inner + group * args.size + n]);
        c[n] = to_float<T>(row[inner + (args.groups + group) * args.size + n]);
    }
    const float step = step_size(args, token, head);
    const float decay = expf(-state_rate(args, head) * step);
    float x[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) x[i] = slice < slices ? to_float<T>(row[head * args.vdim + column + i]) : 0.0f;
    __syncthreads();
    float y[4] = {};
    if (slice < slices) {
        for (uint32_t first = slice; first < args.size; first += kBatch * slices) {
            if (first != slice) load_batch(first);
#pragma unroll
            for (uint32_t i = 0; i < kBatch; ++i) {
                const uint32_t n = first + i * slices;
                if (n < args.size) {
                    const float weight = step * b[n];
                    float4 value = held[i];
                    value.x = fmaf(weight, x[0], value.x * decay);
                    value.y = fmaf(weight, x[1], value.y * decay);
                    value.z = fmaf(weight, x[2], value.z * decay);
                    value.w = fmaf(weight, x[3], value.w * decay);
                    state[static_cast<size_t>(n) * quads] = value;
                    const float read = c[n];
                    y[0] = fmaf(read, value.x, y[0]);
                    y[1] = fmaf(read, value.y, y[1]);
                    y[2] = fmaf(read, value.z, y[2]);
                    y[3] = fmaf(read, value.w, y[3]);
                }
            }
        }
        *reinterpret_cast<float4*>(partial + slice * args.vdim + column) = make_float4(y[0], y[1], y[2], y[3]);
    }
    __syncthreads();
    const float skip = __bfloat162float(args.skip[head]);
    for (uint32_t v = threadIdx.x; v < args.vdim; v += kDecodeThreads) {
        float sum = skip * to_float<T>(row[head * args.vdim + v]);
        for (uint32_t s = 0; s < slices; ++s) sum += partial[s * args.vdim + v];
        args.out[token * inner + head * args.vdim + v] = from_float<T>(sum);
    }
}

// ------------------------------------------------------------------------------------------------ token by token

constexpr uint32_t kScanThreads = 256;
constexpr uint32_t kScanColumns = 32;
constexpr uint32_t kScanTokens = 8;

// One CTA per segment, head and 32 columns of the state, any sizes, either activation type.  A warp owns four columns, its
// lanes eight interleaved slices of the rows, held in registers over the whole segment.
template <typename T, int ROWS>
__global__ void __launch_bounds__(kScanThreads)
state_space_scan_kernel(const StateSpaceArgs<T> args, uint32_t column_blocks) {
    pdl_launch_dependents();
    extern __shared__ float shared[];
    float* b = shared;                                    // [tokens][size]
    float* c = b + kScanTokens * args.size;               // [tokens][size]
    __shared__ float x[kScanTokens][kScanColumns], y[kScanTokens][kScanColumns], decays[kScanTokens], steps[kScanTokens];
    pdl_wait();
    const uint32_t block = blockIdx.x % column_blocks;
    const uint32_t head = blockIdx.x / column_blocks % args.heads;
    const uint32_t segment = blockIdx.x / column_blocks / args.heads;
    const size_t slot = args.segments.slots[segment];
    if (slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t begin = args.segments.offsets != nullptr ? args.segments.offsets[segment] : segment;
    const uint32_t stop = args.segments.offsets != nullptr ? args.segments.offsets[segment + 1] : segment + 1;
    const uint32_t end = stop < args.segments.num_tokens ? stop : static_cast<uint32_t>(args.segments.num_tokens);
    const uint32_t group = head / (args.heads / args.groups);
    const size_t inner = static_cast<size_t>(args.heads) * args.vdim;
    const uint32_t column0 = block * kScanColumns;
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t slice = lane & 7;
    const uint32_t local = (threadIdx.x >> 5) * 4 + (lane >> 3);
    const uint32_t column = column0 + local;
    const bool live = column < args.vdim;
    float* state = state_of(args, slot, head) + column;
    float held[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const uint32_t n = slice + 8 * i;
        held[i] = live && n < args.size ? state[static_cast<size_t>(n) * args.vdim] : 0.0f;
    }
    const float rate = state_rate(args, head);
    const float skip = __bfloat162float(args.skip[head]);
    for (uint32_t base = begin; base < end; base += kScanTokens) {
        const uint32_t count = end - base < kScanTokens ? end - base : kScanTokens;
        __syncthreads();
        for (uint32_t item = threadIdx.x; item < count * args.size; item += kScanThreads) {
            const T* row = args.mixed + static_cast<size_t>(base + item / args.size) * args.mixed_pitch + inner;
            b[item] = to_float<T>(row[group * args.size + item % args.size]);
            c[item] = to_float<T>(row[(args.groups + group) * args.size + item % args.size]);
        }
        for (uint32_t item = threadIdx.x; item < count * kScanColumns; item += kScanThreads) {
            const uint32_t v = column0 + item % kScanColumns;
            x[item / kScanColumns][item % kScanColumns] =
                v < args.vdim ? to_float<T>(args.mixed[static_cast<size_t>(base + item / kScanColumns) * args.mixed_pitch +
                                                       head * args.vdim + v])
                              : 0.0f;
        }
        if (threadIdx.x < count) {
            const float step = step_size(args, base + threadIdx.x, head);
            steps[threadIdx.x] = step;
            decays[threadIdx.x] = expf(-rate * step);
        }
        __syncthreads();
        for (uint32_t t = 0; t < count; ++t) {
            const float decay = decays[t];
            const float input = x[t][local];
            const float weighted = steps[t] * input;
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < ROWS; ++i) {
                const uint32_t n = slice + 8 * i;
                if (n < args.size) {
                    held[i] = fmaf(b[t * args.size + n], weighted, held[i] * decay);
                    sum = fmaf(c[t * args.size + n], held[i], sum);
                }
            }
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            sum += __shfl_xor_sync(0xffffffffu, sum, 2);
            sum += __shfl_xor_sync(0xffffffffu, sum, 4);
            if (slice == 0) y[t][local] = fmaf(skip, input, sum);
        }
        __syncthreads();
        for (uint32_t item = threadIdx.x; item < count * kScanColumns; item += kScanThreads) {
            const uint32_t v = column0 + item % kScanColumns;
            if (v < args.vdim) {
                args.out[static_cast<size_t>(base + item / kScanColumns) * inner + head * args.vdim + v] =
                    from_float<T>(y[item / kScanColumns][item % kScanColumns]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const uint32_t n = slice + 8 * i;
        if (live && n < args.size) state[static_cast<size_t>(n) * args.vdim] = held[i];
    }
}

template <typename T>
cudaError_t launch_decode(cudaStream_t stream, const StateSpaceLaunch& launch, size_t tokens) {
    const uint32_t slices = kDecodeThreads / (launch.vdim / 4);
    const size_t shared =
        ((2 * static_cast<size_t>(launch.size) + 3) / 4 * 4 + static_cast<size_t>(slices) * launch.vdim) * sizeof(float);
    return launch_kernel(state_space_decode_kernel<T>, static_cast<unsigned int>(tokens * launch.heads), kDecodeThreads,
                         shared, stream, 1, state_space_args<T>(launch));
}

template <typename T>
cudaError_t launch_scan(cudaStream_t stream, const StateSpaceLaunch& launch) {
    const uint32_t column_blocks = (launch.vdim + kScanColumns - 1) / kScanColumns;
    const size_t shared = 2 * kScanTokens * static_cast<size_t>(launch.size) * sizeof(float);
    void (*kernel)(const StateSpaceArgs<T>, uint32_t) = nullptr;
    if (launch.size <= 64) {
        kernel = state_space_scan_kernel<T, 8>;
    } else if (launch.size <= 128) {
        kernel = state_space_scan_kernel<T, 16>;
    } else if (launch.size <= 256) {
        kernel = state_space_scan_kernel<T, 32>;
    } else if (launch.size <= kStateSpaceMaxSize) {
        kernel = state_space_scan_kernel<T, 64>;
    } else {
        return cudaErrorInvalidValue;
    }
    const size_t blocks = launch.segments.num_segments * launch.heads * column_blocks;
    return launch_kernel(kernel, static_cast<unsigned int>(blocks), kScanThreads, shared, stream, 1,
                         state_space_args<T>(launch), column_blocks);
}

// ------------------------------------------------------------------------------------------------ gated norm

// One warp per row and part where a part fits the registers of a warp (HELD vectors per lane), else one CTA.
template <typename T, int VEC, int HELD>
__global__ void __launch_bounds__(512)
gated_group_norm_kernel(const T* __restrict__ y, const T* __restrict__ z, size_t z_pitch,
                        const __nv_bfloat16* __restrict__ norm, T* __restrict__ out, size_t out_pitch, size_t tokens,
                        size_t width, uint32_t groups, float eps) {
    pdl_launch_dependents();
    __shared__ float scratch[16];
    pdl_wait();
    const size_t part = width / groups;
    auto gated = [&](size_t token, size_t column, float (&value)[VEC]) {
        float gate[VEC];
        load_values<VEC>(y + token * width + column, value);
        load_values<VEC>(z + token * z_pitch + column, gate);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] *= gate[i] * sigmoid_of<T>(gate[i]);
    };
    auto emit = [&](size_t token, size_t column, float (&value)[VEC], float scale) {
        float weight[VEC];
        load_values<VEC>(norm + column, weight);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] *= scale * weight[i];
        store_values<VEC>(out + token * out_pitch + column, value);
    };
    float sum = 0.0f;
    if constexpr (HELD > 0) {
        const size_t item = static_cast<size_t>(blockIdx.x) * (blockDim.x / 32) + threadIdx.x / 32;
        if (item >= tokens * groups) {
            return;
        }
        const size_t token = item / groups;
        const size_t first = item % groups * part;
        const size_t mine = (threadIdx.x & 31) * VEC;
        float held[HELD][VEC];
#pragma unroll
        for (int step = 0; step < HELD; ++step) {
            const size_t column = mine + step * 32 * VEC;
            if (column < part) gated(token, first + column, held[step]);
        }
#pragma unroll
        for (int step = 0; step < HELD; ++step) {
            if (mine + step * 32 * VEC < part) {
#pragma unroll
                for (int i = 0; i < VEC; ++i) sum = fmaf(held[step][i], held[step][i], sum);
            }
        }
        const float scale = inverse_rms(warp_sum(sum), part, eps);
#pragma unroll
        for (int step = 0; step < HELD; ++step) {
            const size_t column = mine + step * 32 * VEC;
            if (column < part) emit(token, first + column, held[step], scale);
        }
    } else {
        const size_t token = blockIdx.x / groups;
        const size_t first = blockIdx.x % groups * part;
        const size_t mine = threadIdx.x * VEC;
        float held[VEC];                       // the thread's first vector stays in registers
        for (size_t column = mine; column < part; column += blockDim.x * VEC) {
            float value[VEC];
            gated(token, first + column, value);
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                sum = fmaf(value[i], value[i], sum);
                if (column == mine) held[i] = value[i];
            }
        }
        const float scale = inverse_rms(block_sum(sum, scratch), part, eps);
        for (size_t column = mine; column < part; column += blockDim.x * VEC) {
            if (column != mine) gated(token, first + column, held);
            emit(token, first + column, held, scale);
        }
    }
}

}  // namespace

cudaError_t launch_channel_conv(cudaStream_t stream, const ChannelConvLaunch& launch) {
    return launch.type == Activation::kF32 ? launch_conv<float>(stream, launch)
                                           : launch_conv<__nv_bfloat16>(stream, launch);
}

cudaError_t launch_state_space(cudaStream_t stream, const StateSpaceLaunch& launch) {
    const bool f32 = launch.type == Activation::kF32;
    StateSpaceLaunch rest = launch;
    const bool decode = launch.vdim % 4 == 0 && launch.vdim / 4 <= kDecodeThreads && launch.record.offset % 16 == 0 &&
                        launch.record.stride % 16 == 0 && aligned_to(launch.record.base, 16);
    if (launch.decode_tokens > 0 && decode) {
        const cudaError_t status = f32 ? launch_decode<float>(stream, launch, launch.decode_tokens)
                                       : launch_decode<__nv_bfloat16>(stream, launch, launch.decode_tokens);
        if (status != cudaSuccess || launch.decode_tokens == launch.segments.num_segments) return status;
        // segment offsets are absolute token indices, so the remaining segments are simply a later start
        rest.segments.offsets += launch.decode_tokens;
        rest.segments.slots += launch.decode_tokens;
        rest.segments.num_segments -= launch.decode_tokens;
    }
    if (option(kOptStateSpacePrompt) == 0 && state_space_chunk_supports(rest)) {
        return launch_state_space_chunk(stream, rest);
    }
    return f32 ? launch_scan<float>(stream, rest) : launch_scan<__nv_bfloat16>(stream, rest);
}

cudaError_t launch_gated_group_norm(cudaStream_t stream, const GatedGroupNormLaunch& launch) {
    const size_t part = launch.width / launch.groups;
    const bool vector = part % 8 == 0 && launch.z_pitch % 8 == 0 && launch.out_pitch % 8 == 0 && aligned_to(launch.y, 16) &&
                        aligned_to(launch.z, 16) && aligned_to(launch.norm, 16) && aligned_to(launch.out, 16);
    const size_t vectors = vector ? part / 8 : part;
    const size_t items = launch.tokens * launch.groups;
    const bool warps = vector && vectors <= 64;
    const unsigned int threads = warps ? 128 : static_cast<unsigned int>(std::min<size_t>((vectors + 31) / 32 * 32, 512));
    const unsigned int blocks = static_cast<unsigned int>(warps ? (items + 3) / 4 : items);
    auto go = [&](auto* typed, auto kernel) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(kernel, blocks, threads, 0, stream, 1, static_cast<const T*>(launch.y),
                             static_cast<const T*>(launch.z), launch.z_pitch, static_cast<const __nv_bfloat16*>(launch.norm),
                             static_cast<T*>(launch.out), launch.out_pitch, launch.tokens, launch.width, launch.groups,
                             launch.eps);
    };
    auto sized = [&](auto* typed) {
        using T = std::remove_pointer_t<decltype(typed)>;
        if (!vector) return go(typed, gated_group_norm_kernel<T, 1, 0>);
        if (!warps) return go(typed, gated_group_norm_kernel<T, 8, 0>);
        return vectors <= 32 ? go(typed, gated_group_norm_kernel<T, 8, 1>) : go(typed, gated_group_norm_kernel<T, 8, 2>);
    };
    return launch.type == Activation::kF32 ? sized(static_cast<float*>(nullptr))
                                           : sized(static_cast<__nv_bfloat16*>(nullptr));
}

}  // namespace lfm25
