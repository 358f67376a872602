// Row kernels of the layer stack: residual sum + two norms + input convolution in one pass, the final norm on selected
// rows, the polynomial activation, and greedy sampling.
#include <math.h>

#include <algorithm>

#include "launch.h"
#include "stack_common.cuh"

namespace lfm25 {

namespace {

constexpr uint32_t kThreads = 256;
constexpr size_t kMaxSharedBytes = 227 * 1024;

struct ResidualNormConvArgs {
    StackSegments segments;
    const float* residual;
    const uint32_t* token_ids;
    const __nv_bfloat16* embedding;
    size_t vocab;
    const __nv_bfloat16* mixer_norm;
    const __nv_bfloat16* ff_norm;
    const __nv_bfloat16* conv;
    uint32_t taps;
    uint32_t tile_rows;
    StackRecord record;
    float* residual_out;
    size_t width;
    float eps;
};

// One row of the residual stream before the layer: x[c .. c + VEC)
template <typename T, int VEC>
__device__ __forceinline__ void residual_values(const ResidualNormConvArgs& args, const T* update,
                                                const __nv_bfloat16* embedding_row, size_t row, size_t channel,
                                                float (&value)[VEC]) {
    if (args.embedding != nullptr) {
        if (embedding_row != nullptr) {
            load_values<VEC>(embedding_row + channel, value);
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) value[i] = 0.0f;
        }
    } else {
        load_values<VEC>(args.residual + row * args.width + channel, value);
    }
    if (update != nullptr) {
        float add[VEC];
        load_values<VEC>(update + row * args.width + channel, add);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] += add[i];
    }
}

// One CTA per tile of tokens of one segment.  First the norms: every row the tile needs -- its own, the taps - 1 before
// it, and for the segment's first tile the last taps - 1 of the segment -- is normalised once into shared memory, rounded
// to the activation type as the stored history is.  Then the convolution per channel from shared memory and, for the
// first tokens of the segment, the record.  Only the segment's first tile touches the record: it reads it for its own
// first rows and replaces it afterwards, so no other CTA depends on the order.
// GROUP threads share a row: the whole CTA when a tile is one row (decode), one warp otherwise.
// HELD: a row fits the registers of its threads (one vector each), so that it is read once.
// TAPS: number of taps known at compile time (0 = any), whose weights and window then stay in registers.
template <typename T, int VEC, int GROUP, bool HELD, int TAPS>
__global__ void __launch_bounds__(kThreads, GROUP == 32 ? 3 : 1)
residual_norm_conv_kernel(const ResidualNormConvArgs args, const T* __restrict__ update, T* __restrict__ mixed_out,
                          T* __restrict__ ff_out) {
    pdl_launch_dependents();
    pdl_wait();
    static_assert(!HELD || GROUP == kThreads, "a row is held by a whole CTA");
    constexpr int kHeld = 1;
    extern __shared__ __align__(16) unsigned char shared_raw[];
    __shared__ float scratch[kThreads / 32];
    T* rows = reinterpret_cast<T*>(shared_raw);      // [taps - 1 + tile_rows][width]
    const SegmentTile tile = locate_tile(args.segments, args.tile_rows, blockIdx.x);
    if (tile.count == 0) {
        return;
    }
    const uint32_t history = args.taps - 1;
    const size_t width = args.width;
    const bool first_tile = tile.first == tile.begin;
    const size_t slot = args.segments.slots[tile.segment];
    if (slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t group = threadIdx.x / GROUP;
    const uint32_t lane = threadIdx.x % GROUP;
    // rows of shared memory: [0, history) the tokens before the tile (first tile: the segment's last tokens, where
    // they are not in the tile itself), then the tile
    for (uint32_t index = group; index < history + tile.count; index += kThreads / GROUP) {
        uint32_t token;
        bool own = false;
        if (index >= history) {
            token = tile.first + (index - history);
            own = true;
        } else if (first_tile) {
            if (tile.end < tile.first + tile.count + (history - index)) {
                continue;       // end - (history - index) lies in the tile or before the segment
            }
            token = tile.end - (history - index);
        } else {
            token = tile.first - (history - index);     // tile_rows >= history: inside the segment
        }
        const __nv_bfloat16* embedding_row = nullptr;
        if (args.embedding != nullptr) {
            const size_t id = args.token_ids[token];
            embedding_row = id < args.vocab ? args.embedding + id * width : nullptr;
        }
        float sum = 0.0f;
        float held[kHeld][VEC];           // the row between the two passes, when it fits
        auto accumulate = [&](size_t channel, float (&value)[VEC]) {
            residual_values<T, VEC>(args, update, embedding_row, token, channel, value);
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum = fmaf(value[i], value[i], sum);
        };
        auto emit = [&](size_t channel, const float (&value)[VEC], float scale) {
            float weight[VEC], result[VEC];
            load_values<VEC>(args.mixer_norm + channel, weight);
#pragma unroll
            for (int i = 0; i < VEC; ++i) result[i] = value[i] * scale * weight[i];
            store_values<VEC>(rows + index * width + channel, result);
            if (!own) {
                return;
            }
            store_values<VEC>(args.residual_out + static_cast<size_t>(token) * width + channel, value);
            if (args.ff_norm != nullptr) {
                load_values<VEC>(args.ff_norm + channel, weight);
#pragma unroll
                for (int i = 0; i < VEC; ++i) result[i] = value[i] * scale * weight[i];
                store_values<VEC>(ff_out + static_cast<size_t>(token) * width + channel, result);
            }
        };
        if constexpr (HELD) {
#pragma unroll
            for (int step = 0; step < kHeld; ++step) {
                const size_t channel = (step * GROUP + lane) * VEC;
                if (channel < width) accumulate(channel, held[step]);
            }
        } else {
            for (size_t channel = lane * VEC; channel < width; channel += GROUP * VEC) accumulate(channel, held[0]);
        }
        sum = GROUP == 32 ? warp_sum(sum) : block_sum(sum, scratch);
        const float scale = inverse_rms(sum, width, args.eps);
        if constexpr (HELD) {
#pragma unroll
            for (int step = 0; step < kHeld; ++step) {
                const size_t channel = (step * GROUP + lane) * VEC;
                if (channel < width) emit(channel, held[step], scale);
            }
        } else {
            for (size_t channel = lane * VEC; channel < width; channel += GROUP * VEC) {
                residual_values<T, VEC>(args, update, embedding_row, token, channel, held[0]);
                emit(channel, held[0], scale);
            }
        }
    }
    __syncthreads();

    T* record = reinterpret_cast<T*>(static_cast<unsigned char*>(args.record.base) + slot * args.record.stride +
                                     args.record.offset);
    for (size_t channel = threadIdx.x * VEC; channel < width; channel += kThreads * VEC) {
        // the input `back` tokens before row `row` of the tile: in shared memory, or in the record (whose last row is
        // the token before the segment)
        auto load_input = [&](uint32_t row, uint32_t back, float (&value)[VEC]) {
            const uint32_t offset = tile.first - tile.begin + row;     // of the token in its segment
            if (back > offset) {
                load_values<VEC>(record + (history - (back - offset)) * width + channel, value);
            } else {
                load_values<VEC>(rows + (history + row - back) * width + channel, value);
            }
        };
        if constexpr (TAPS > 0) {
            float tap[TAPS][VEC], window[TAPS][VEC];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) load_values<VEC>(args.conv + j * width + channel, tap[j]);
#pragma unroll
            for (int j = 1; j < TAPS; ++j) load_input(0, TAPS - j, window[j]);
            for (uint32_t row = 0; row < tile.count; ++row) {
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) {
#pragma unroll
                    for (int i = 0; i < VEC; ++i) window[j][i] = window[j + 1][i];
                }
                load_values<VEC>(rows + (history + row) * width + channel, window[TAPS - 1]);
                float sum[VEC];
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    sum[i] = 0.0f;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) sum[i] = fmaf(tap[j][i], window[j][i], sum[i]);
                    sum[i] += window[TAPS - 1][i];
                }
                store_values<VEC>(mixed_out + static_cast<size_t>(tile.first + row) * width + channel, sum);
            }
        } else {
            for (uint32_t row = 0; row < tile.count; ++row) {
                float sum[VEC], value[VEC], tap[VEC];
#pragma unroll
                for (int i = 0; i < VEC; ++i) sum[i] = 0.0f;
                for (uint32_t j = 0; j < args.taps; ++j) {
                    load_input(row, history - j, value);
                    load_values<VEC>(args.conv + j * width + channel, tap);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) sum[i] = fmaf(tap[i], value[i], sum[i]);
                }
                load_values<VEC>(rows + (history + row) * width + channel, value);
#pragma unroll
                for (int i = 0; i < VEC; ++i) value[i] += sum[i];
                store_values<VEC>(mixed_out + static_cast<size_t>(tile.first + row) * width + channel, value);
            }
        }
        if (first_tile) {
            // the same thread has read this channel's history above; ascending order only reads rows not yet written
            const uint32_t length = tile.end - tile.begin;
            for (uint32_t i = 0; i < history; ++i) {
                const uint32_t back = history - i;                     // distance from the segment's end
                float value[VEC];
                if (back > length) {
                    load_values<VEC>(record + (history - (back - length)) * width + channel, value);
                } else if (length - back < tile.count) {
                    load_values<VEC>(rows + (history + length - back) * width + channel, value);
                } else {
                    load_values<VEC>(rows + i * width + channel, value);
                }
                store_values<VEC>(record + i * width + channel, value);
            }
        }
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
residual_norm_rows_kernel(const float* __restrict__ residual, const T* __restrict__ update,
                          const __nv_bfloat16* __restrict__ weight, const uint32_t* __restrict__ rows,
                          T* __restrict__ out, size_t num_tokens, size_t width, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[kThreads / 32];
    const size_t row = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
    if (row >= num_tokens) {
        return;
    }
    float sum = 0.0f;
    for (size_t channel = threadIdx.x * VEC; channel < width; channel += kThreads * VEC) {
        float value[VEC], add[VEC];
        load_values<VEC>(residual + row * width + channel, value);
        load_values<VEC>(update + row * width + channel, add);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            value[i] += add[i];
            sum = fmaf(value[i], value[i], sum);
        }
    }
    const float scale = inverse_rms(block_sum(sum, scratch), width, eps);
    for (size_t channel = threadIdx.x * VEC; channel < width; channel += kThreads * VEC) {
        float value[VEC], add[VEC], norm[VEC];
        load_values<VEC>(residual + row * width + channel, value);
        load_values<VEC>(update + row * width + channel, add);
        load_values<VEC>(weight + channel, norm);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] = (value[i] + add[i]) * scale * norm[i];
        store_values<VEC>(out + blockIdx.x * width + channel, value);
    }
}

struct PostNormArgs {
    const float* residual;
    const __nv_bfloat16* post_norm;
    const uint32_t* token_ids;
    const __nv_bfloat16* embedding;
    size_t vocab;
    const __nv_bfloat16* norm;
    const uint32_t* rows;
    float* residual_out;
    size_t num_tokens;
    size_t width;
    float shift;
    float eps;
};

// One CTA per row.  HELD: vectors of the row that each thread keeps in registers, so that everything is read once; 0: any
// width, the row is read again for every pass (residual_out then holds the sum between the passes).
template <typename T, int VEC, int HELD>
__global__ void __launch_bounds__(512)
residual_post_norm_kernel(const PostNormArgs args, const T* __restrict__ update, T* __restrict__ out) {
    pdl_launch_dependents();
    __shared__ float scratch[16];
    pdl_wait();
    const size_t row = args.rows != nullptr ? args.rows[blockIdx.x] : blockIdx.x;
    if (row >= args.num_tokens) {
        return;
    }
    const size_t width = args.width;
    const size_t step = static_cast<size_t>(blockDim.x) * VEC;
    const __nv_bfloat16* embedding_row = nullptr;
    if (args.embedding != nullptr) {
        const size_t id = args.token_ids[row];
        embedding_row = id < args.vocab ? args.embedding + id * width : nullptr;
    }
    auto load_residual = [&](size_t channel, float (&value)[VEC]) {
        if (args.embedding == nullptr) {
            load_values<VEC>(args.residual + row * width + channel, value);
        } else if (embedding_row != nullptr) {
            load_values<VEC>(embedding_row + channel, value);
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) value[i] = 0.0f;
        }
    };
    auto load_weight = [&](const __nv_bfloat16* weight, size_t channel, float (&value)[VEC]) {
        load_values<VEC>(weight + channel, value);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] += args.shift;
    };
    auto add_squares = [](const float (&value)[VEC], float& sum) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) sum = fmaf(value[i], value[i], sum);
    };
    auto write_residual = [&](size_t channel, const float (&value)[VEC]) {
        if (args.residual_out != nullptr) store_values<VEC>(args.residual_out + blockIdx.x * width + channel, value);
    };
    auto write_out = [&](size_t channel, float (&value)[VEC], float scale) {
        float weight[VEC];
        load_weight(args.norm, channel, weight);
#pragma unroll
        for (int i = 0; i < VEC; ++i) value[i] *= scale * weight[i];
        store_values<VEC>(out + blockIdx.x * width + channel, value);
    };
    if constexpr (HELD > 0) {
        float held[HELD][VEC];
#pragma unroll
        for (int part = 0; part < HELD; ++part) {
            const size_t channel = part * step + threadIdx.x * VEC;
            if (channel < width) load_residual(channel, held[part]);
        }
        if (update != nullptr) {
            float add[HELD][VEC], sum = 0.0f;
#pragma unroll
            for (int part = 0; part < HELD; ++part) {
                const size_t channel = part * step + threadIdx.x * VEC;
                if (channel < width) {
                    load_values<VEC>(update + row * width + channel, add[part]);
                    add_squares(add[part], sum);
                }
            }
            const float scale = inverse_rms(block_sum(sum, scratch), width, args.eps);
#pragma unroll
            for (int part = 0; part < HELD; ++part) {
                const size_t channel = part * step + threadIdx.x * VEC;
                if (channel < width) {
                    float weight[VEC];
                    load_weight(args.post_norm, channel, weight);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) held[part][i] += add[part][i] * scale * weight[i];
                }
            }
        }
        float sum = 0.0f;
#pragma unroll
        for (int part = 0; part < HELD; ++part) {
            const size_t channel = part * step + threadIdx.x * VEC;
            if (channel < width) {
                write_residual(channel, held[part]);
                add_squares(held[part], sum);
            }
        }
        if (out == nullptr) {
            return;
        }
        const float scale = inverse_rms(block_sum(sum, scratch), width, args.eps);
#pragma unroll
        for (int part = 0; part < HELD; ++part) {
            const size_t channel = part * step + threadIdx.x * VEC;
            if (channel < width) write_out(channel, held[part], scale);
        }
    } else {
        float post = 0.0f;
        if (update != nullptr) {
            float sum = 0.0f;
            for (size_t channel = threadIdx.x * VEC; channel < width; channel += step) {
                float add[VEC];
                load_values<VEC>(update + row * width + channel, add);
                add_squares(add, sum);
            }
            post = inverse_rms(block_sum(sum, scratch), width, args.eps);
        }
        auto sum_of = [&](size_t channel, float (&value)[VEC]) {
            load_residual(channel, value);
            if (update != nullptr) {
                float add[VEC], weight[VEC];
                load_values<VEC>(update + row * width + channel, add);
                load_weight(args.post_norm, channel, weight);
#pragma unroll
                for (int i = 0; i < VEC; ++i) value[i] += add[i] * post * weight[i];
            }
        };
        float sum = 0.0f, value[VEC];
        for (size_t channel = threadIdx.x * VEC; channel < width; channel += step) {
            sum_of(channel, value);
            add_squares(value, sum);
        }
        const float scale = inverse_rms(block_sum(sum, scratch), width, args.eps);
        for (size_t channel = threadIdx.x * VEC; channel < width; channel += step) {
            sum_of(channel, value);
            write_residual(channel, value);       // the thread that reads this channel again is this one
            if (out != nullptr) write_out(channel, value, scale);
        }
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
squared_relu_kernel(T* __restrict__ z, size_t count) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t at = (static_cast<size_t>(blockIdx.x) * kThreads + threadIdx.x) * VEC;
    if (at < count) {
        float value[VEC];
        load_values<VEC>(z + at, value);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float positive = fmaxf(value[i], 0.0f);
            value[i] = positive * positive;
        }
        store_values<VEC>(z + at, value);
    }
}

struct PolyCoefficients {
    float a, b, c, e;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
poly_norm_kernel(const T* __restrict__ z, size_t z_pitch, T* __restrict__ out, size_t out_pitch, size_t width,
                 size_t pad, PolyCoefficients coefficients, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[3][kThreads / 32];
    const T* source = z + blockIdx.x * z_pitch;
    T* target = out + blockIdx.x * out_pitch;
    float sum1 = 0.0f, sum2 = 0.0f, sum3 = 0.0f;
    for (size_t column = threadIdx.x * VEC; column < width; column += kThreads * VEC) {
        float value[VEC];
        load_values<VEC>(source + column, value);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float square = value[i] * value[i];
            const float cube = square * value[i];
            sum1 += square;
            sum2 = fmaf(square, square, sum2);
            sum3 = fmaf(cube, cube, sum3);
        }
    }
    // the three sums share two barriers
    sum1 = warp_sum(sum1);
    sum2 = warp_sum(sum2);
    sum3 = warp_sum(sum3);
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    if (lane == 0) {
        scratch[0][warp] = sum1;
        scratch[1][warp] = sum2;
        scratch[2][warp] = sum3;
    }
    __syncthreads();
    constexpr uint32_t kWarps = kThreads / 32;
    sum1 = warp_sum(lane < kWarps ? scratch[0][lane] : 0.0f);
    sum2 = warp_sum(lane < kWarps ? scratch[1][lane] : 0.0f);
    sum3 = warp_sum(lane < kWarps ? scratch[2][lane] : 0.0f);
    const float a = coefficients.a * inverse_rms(sum1, width, eps);
    const float b = coefficients.b * inverse_rms(sum2, width, eps);
    const float c = coefficients.c * inverse_rms(sum3, width, eps);
    for (size_t column = threadIdx.x * VEC; column < width; column += kThreads * VEC) {
        float value[VEC];
        load_values<VEC>(source + column, value);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float square = value[i] * value[i];
            value[i] = a * value[i] + b * square + c * (square * value[i]) + coefficients.e;
        }
        store_values<VEC>(target + column, value);
    }
    for (size_t column = width + threadIdx.x; column < width + pad; column += kThreads) {
        target[column] = from_float<T>(0.0f);
    }
}

// Larger value first, then the lower index; NaN counts as smaller than everything.
struct Candidate {
    float value;
    uint32_t index;
};
__device__ __forceinline__ bool better(const Candidate& a, const Candidate& b) {
    return a.value > b.value || (a.value == b.value && a.index < b.index);
}
__device__ __forceinline__ Candidate warp_best(Candidate best) {
#pragma unroll
    for (uint32_t delta = 16; delta > 0; delta >>= 1) {
        Candidate other;
        other.value = __shfl_xor_sync(0xffffffffu, best.value, delta);
        other.index = __shfl_xor_sync(0xffffffffu, best.index, delta);
        if (better(other, best)) best = other;
    }
    return best;
}

constexpr uint32_t kArgmaxThreads = 512;
template <typename T, int VEC>
__global__ void __launch_bounds__(kArgmaxThreads)
argmax_kernel(const T* __restrict__ logits, size_t pitch, uint32_t* __restrict__ sampled, uint32_t vocab) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ Candidate held[kArgmaxThreads / 32];
    const T* row = logits + blockIdx.x * pitch;
    Candidate best = {-INFINITY, 0xffffffffu};
    for (uint32_t column = threadIdx.x * VEC; column < vocab; column += kArgmaxThreads * VEC) {
        float value[VEC];
        load_values<VEC>(row + column, value);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            if (value[i] > best.value || (value[i] == best.value && column + i < best.index)) {
                best = {value[i], column + i};
            }
        }
    }
    best = warp_best(best);
    const uint32_t lane = threadIdx.x & 31;
    if (lane == 0) {
        held[threadIdx.x >> 5] = best;
    }
    __syncthreads();
    if (threadIdx.x < 32) {
        best = lane < kArgmaxThreads / 32 ? held[lane] : Candidate{-INFINITY, 0xffffffffu};
        best = warp_best(best);
        if (lane == 0) {
            sampled[blockIdx.x] = best.index < vocab ? best.index : 0u;
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(kThreads)
export_logits_kernel(const T* __restrict__ logits, size_t pitch, float* __restrict__ out, size_t vocab, float softcap) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t blocks = (vocab + kThreads - 1) / kThreads;
    const size_t row = blockIdx.x / blocks;
    const size_t column = blockIdx.x % blocks * kThreads + threadIdx.x;
    if (column < vocab) {
        const float value = to_float<T>(logits[row * pitch + column]);
        out[row * vocab + column] = softcap > 0.0f ? softcap * tanhf(value / softcap) : value;
    }
}

// ------------------------------------------------------------------------------------------ plain matrix product

constexpr uint32_t kTile = 64;
constexpr uint32_t kDepth = 16;

// 64 x 64 outputs per CTA, 4 x 4 per thread, products and sums in f32
template <typename T>
__global__ void __launch_bounds__(256)
linear_simt_kernel(const T* __restrict__ x, const __nv_bfloat16* __restrict__ weight, T* __restrict__ y, size_t m,
                   size_t n, size_t k) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float x_tile[kDepth][kTile + 4];
    __shared__ float w_tile[kDepth][kTile + 4];
    const size_t columns = (n + kTile - 1) / kTile;
    const size_t row0 = blockIdx.x / columns * kTile;
    const size_t column0 = blockIdx.x % columns * kTile;
    const uint32_t tx = threadIdx.x & 15;
    const uint32_t ty = threadIdx.x >> 4;
    float sum[4][4] = {};
    for (size_t depth = 0; depth < k; depth += kDepth) {
#pragma unroll
        for (uint32_t part = 0; part < kTile * kDepth / 256; ++part) {
            const uint32_t item = threadIdx.x + part * 256;
            const uint32_t row = item / kDepth;
            const uint32_t inner = item % kDepth;
            const bool inside = depth + inner < k;
            x_tile[inner][row] =
                inside && row0 + row < m ? to_float<T>(x[(row0 + row) * k + depth + inner]) : 0.0f;
            w_tile[inner][row] =
                inside && column0 + row < n ? __bfloat162float(weight[(column0 + row) * k + depth + inner]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (uint32_t inner = 0; inner < kDepth; ++inner) {
            float a[4], b[4];
#pragma unroll
            for (uint32_t i = 0; i < 4; ++i) {
                a[i] = x_tile[inner][ty * 4 + i];
                b[i] = w_tile[inner][tx * 4 + i];
            }
#pragma unroll
            for (uint32_t i = 0; i < 4; ++i) {
#pragma unroll
                for (uint32_t j = 0; j < 4; ++j) sum[i][j] = fmaf(a[i], b[j], sum[i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (uint32_t i = 0; i < 4; ++i) {
#pragma unroll
        for (uint32_t j = 0; j < 4; ++j) {
            const size_t row = row0 + ty * 4 + i;
            const size_t column = column0 + tx * 4 + j;
            if (row < m && column < n) {
                y[row * n + column] = from_float<T>(sum[i][j]);
            }
        }
    }
}

template <typename T>
cudaError_t launch_rnc(cudaStream_t stream, const ResidualNormConvLaunch& launch) {
    ResidualNormConvArgs args;
    args.segments = launch.segments;
    args.residual = launch.residual;
    args.token_ids = launch.token_ids;
    args.embedding = static_cast<const __nv_bfloat16*>(launch.embedding);
    args.vocab = launch.vocab;
    args.mixer_norm = static_cast<const __nv_bfloat16*>(launch.mixer_norm);
    args.ff_norm = static_cast<const __nv_bfloat16*>(launch.ff_norm);
    args.conv = static_cast<const __nv_bfloat16*>(launch.conv);
    args.taps = launch.taps;
    args.record = launch.record;
    args.residual_out = launch.residual_out;
    args.width = launch.width;
    args.eps = launch.eps;
    const bool single = launch.segments.offsets == nullptr;
    const size_t history = launch.taps - 1;
    const size_t row_bytes = launch.width * sizeof(T);
    // rows per tile: with their history one row per warp (measured best at three CTAs per SM, more in flight than with
    // rows held in registers), never fewer than the history
    size_t rows = 1;
    if (!single) {
        rows = history >= 4 ? std::max<size_t>(history, 8) : 8 - history;
        while (rows > 1 && rows > history && (rows + history) * row_bytes > kMaxSharedBytes / 2 - 1024) --rows;
    }
    const size_t shared = (rows + history) * row_bytes;
    if (shared > kMaxSharedBytes) {
        return cudaErrorInvalidValue;
    }
    args.tile_rows = static_cast<uint32_t>(rows);
    const bool vector = launch.width % 8 == 0 && aligned_to(launch.residual, 16) && aligned_to(launch.update, 16) &&
                        aligned_to(launch.embedding, 16) && aligned_to(launch.mixer_norm, 16) &&
                        aligned_to(launch.ff_norm, 16) && aligned_to(launch.conv, 16) &&
                        aligned_to(launch.residual_out, 16) && aligned_to(launch.mixed_out, 16) &&
                        aligned_to(launch.ff_out, 16) && aligned_to(launch.record.base, 16) &&
                        launch.record.stride % 16 == 0 && launch.record.offset % 16 == 0;
    void (*kernel)(const ResidualNormConvArgs, const T*, T*, T*) = nullptr;
    if (!vector) {
        kernel = single ? residual_norm_conv_kernel<T, 1, 256, false, 0> : residual_norm_conv_kernel<T, 1, 32, false, 0>;
    } else if (launch.width > 2048) {
        kernel = single ? residual_norm_conv_kernel<T, 8, 256, false, 0> : residual_norm_conv_kernel<T, 8, 32, false, 0>;
    } else if (launch.taps == 4) {
        kernel = single ? residual_norm_conv_kernel<T, 8, 256, true, 4> : residual_norm_conv_kernel<T, 8, 32, false, 4>;
    } else {
        kernel = single ? residual_norm_conv_kernel<T, 8, 256, true, 0> : residual_norm_conv_kernel<T, 8, 32, false, 0>;
    }
    if (shared > 48 * 1024) {
        const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                        cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                        static_cast<int>(shared));
        if (status != cudaSuccess) return status;
    }
    return launch_kernel(kernel, static_cast<unsigned int>(tile_bound(launch.segments, rows)), kThreads, shared, stream,
                         1, args, static_cast<const T*>(launch.update), static_cast<T*>(launch.mixed_out),
                         static_cast<T*>(launch.ff_out));
}

}  // namespace

cudaError_t launch_residual_norm_conv(cudaStream_t stream, const ResidualNormConvLaunch& launch) {
    return launch.type == Activation::kF32 ? launch_rnc<float>(stream, launch)
                                           : launch_rnc<__nv_bfloat16>(stream, launch);
}

cudaError_t launch_residual_norm_rows(cudaStream_t stream, Activation type, const float* residual, const void* update,
                                      const void* weight, const uint32_t* rows, void* out, size_t num_rows,
                                      size_t num_tokens, size_t width, float eps) {
    const bool vector = width % 8 == 0 && aligned_to(residual, 16) && aligned_to(update, 16) && aligned_to(weight, 16) &&
                        aligned_to(out, 16);
    const auto* norm = static_cast<const __nv_bfloat16*>(weight);
    auto go = [&](auto* typed, auto kernel) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(kernel, static_cast<unsigned int>(num_rows), kThreads, 0, stream, 1, residual,
                             static_cast<const T*>(update), norm, rows, static_cast<T*>(out), num_tokens, width, eps);
    };
    if (type == Activation::kF32) {
        float* tag = nullptr;
        return vector ? go(tag, residual_norm_rows_kernel<float, 8>) : go(tag, residual_norm_rows_kernel<float, 1>);
    }
    __nv_bfloat16* tag = nullptr;
    return vector ? go(tag, residual_norm_rows_kernel<__nv_bfloat16, 8>)
                  : go(tag, residual_norm_rows_kernel<__nv_bfloat16, 1>);
}

cudaError_t launch_poly_norm(cudaStream_t stream, Activation type, const void* z, size_t z_pitch, void* out,
                             size_t out_pitch, size_t rows, size_t width, size_t pad, const float coefficients[4],
                             float eps) {
    const PolyCoefficients poly = {coefficients[0], coefficients[1], coefficients[2], coefficients[3]};
    const bool vector = width % 8 == 0 && z_pitch % 8 == 0 && out_pitch % 8 == 0 && aligned_to(z, 16) &&
                        aligned_to(out, 16);
    auto go = [&](auto* typed, auto kernel) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(kernel, static_cast<unsigned int>(rows), kThreads, 0, stream, 1, static_cast<const T*>(z),
                             z_pitch, static_cast<T*>(out), out_pitch, width, pad, poly, eps);
    };
    if (type == Activation::kF32) {
        float* tag = nullptr;
        return vector ? go(tag, poly_norm_kernel<float, 8>) : go(tag, poly_norm_kernel<float, 1>);
    }
    __nv_bfloat16* tag = nullptr;
    return vector ? go(tag, poly_norm_kernel<__nv_bfloat16, 8>) : go(tag, poly_norm_kernel<__nv_bfloat16, 1>);
}

cudaError_t launch_residual_post_norm(cudaStream_t stream, const ResidualPostNormLaunch& launch) {
    PostNormArgs args;
    args.residual = launch.residual;
    args.post_norm = static_cast<const __nv_bfloat16*>(launch.post_norm);
    args.token_ids = launch.token_ids;
    args.embedding = static_cast<const __nv_bfloat16*>(launch.embedding);
    args.vocab = launch.vocab;
    args.norm = static_cast<const __nv_bfloat16*>(launch.norm);
    args.rows = launch.rows;
    args.residual_out = launch.residual_out;
    args.num_tokens = launch.num_tokens;
    args.width = launch.width;
    args.shift = launch.shift;
    args.eps = launch.eps;
    const bool vector = launch.width % 8 == 0 && aligned_to(launch.residual, 16) && aligned_to(launch.update, 16) &&
                        aligned_to(launch.post_norm, 16) && aligned_to(launch.embedding, 16) &&
                        aligned_to(launch.norm, 16) && aligned_to(launch.residual_out, 16) && aligned_to(launch.out, 16);
    const size_t vectors = launch.width / 8;
    const unsigned int threads =
        vector ? static_cast<unsigned int>(std::min<size_t>((vectors + 31) / 32 * 32, 512)) : kThreads;
    const size_t held = (vectors + threads - 1) / threads;
    auto go = [&](auto* typed, auto kernel) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(kernel, static_cast<unsigned int>(launch.num_rows), threads, 0, stream, 1, args,
                             static_cast<const T*>(launch.update), static_cast<T*>(launch.out));
    };
    auto sized = [&](auto* typed) {
        using T = std::remove_pointer_t<decltype(typed)>;
        if (!vector) return go(typed, residual_post_norm_kernel<T, 1, 0>);
        if (held == 1) return go(typed, residual_post_norm_kernel<T, 8, 1>);
        if (held == 2) return go(typed, residual_post_norm_kernel<T, 8, 2>);
        return go(typed, residual_post_norm_kernel<T, 8, 0>);
    };
    return launch.type == Activation::kF32 ? sized(static_cast<float*>(nullptr))
                                           : sized(static_cast<__nv_bfloat16*>(nullptr));
}

cudaError_t launch_squared_relu(cudaStream_t stream, Activation type, void* z, size_t count) {
    const bool vector = count % 8 == 0 && aligned_to(z, 16);
    const size_t per_cta = static_cast<size_t>(kThreads) * (vector ? 8 : 1);
    auto go = [&](auto* typed, auto kernel) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(kernel, static_cast<unsigned int>((count + per_cta - 1) / per_cta), kThreads, 0, stream, 1,
                             static_cast<T*>(z), count);
    };
    if (type == Activation::kF32) {
        float* tag = nullptr;
        return vector ? go(tag, squared_relu_kernel<float, 8>) : go(tag, squared_relu_kernel<float, 1>);
    }
    __nv_bfloat16* tag = nullptr;
    return vector ? go(tag, squared_relu_kernel<__nv_bfloat16, 8>) : go(tag, squared_relu_kernel<__nv_bfloat16, 1>);
}

cudaError_t launch_argmax_rows(cudaStream_t stream, Activation type, const void* logits, size_t pitch,
                               uint32_t* sampled, size_t rows, size_t vocab) {
    const bool vector = vocab % 8 == 0 && pitch % 8 == 0 && aligned_to(logits, 16);
    auto go = [&](auto* typed, auto kernel) {
        using T = std::remove_pointer_t<decltype(typed)>;
        return launch_kernel(kernel, static_cast<unsigned int>(rows), kArgmaxThreads, 0, stream, 1,
                             static_cast<const T*>(logits), pitch, sampled, static_cast<uint32_t>(vocab));
    };
    if (type == Activation::kF32) {
        float* tag = nullptr;
        return vector ? go(tag, argmax_kernel<float, 8>) : go(tag, argmax_kernel<float, 1>);
    }
    __nv_bfloat16* tag = nullptr;
    return vector ? go(tag, argmax_kernel<__nv_bfloat16, 8>) : go(tag, argmax_kernel<__nv_bfloat16, 1>);
}

cudaError_t launch_export_logits(cudaStream_t stream, Activation type, const void* logits, size_t pitch, float* out,
                                 size_t rows, size_t vocab, float softcap) {
    const unsigned int blocks = static_cast<unsigned int>((vocab + kThreads - 1) / kThreads * rows);
    if (type == Activation::kF32) {
        return launch_kernel(export_logits_kernel<float>, blocks, kThreads, 0, stream, 1, static_cast<const float*>(logits),
                             pitch, out, vocab, softcap);
    }
    return launch_kernel(export_logits_kernel<__nv_bfloat16>, blocks, kThreads, 0, stream, 1,
                         static_cast<const __nv_bfloat16*>(logits), pitch, out, vocab, softcap);
}

cudaError_t launch_linear_simt(cudaStream_t stream, Activation type, const void* x, const void* weight, void* y,
                               size_t m, size_t n, size_t k) {
    const size_t tiles = (m + kTile - 1) / kTile * ((n + kTile - 1) / kTile);
    if (tiles == 0 || tiles > 0x7fffffffu) {
        return cudaErrorInvalidValue;
    }
    const auto* w = static_cast<const __nv_bfloat16*>(weight);
    if (type == Activation::kF32) {
        return launch_kernel(linear_simt_kernel<float>, static_cast<unsigned int>(tiles), 256, 0, stream, 1,
                             static_cast<const float*>(x), w, static_cast<float*>(y), m, n, k);
    }
    return launch_kernel(linear_simt_kernel<__nv_bfloat16>, static_cast<unsigned int>(tiles), 256, 0, stream, 1,
                         static_cast<const __nv_bfloat16*>(x), w, static_cast<__nv_bfloat16*>(y), m, n, k);
}

}  // namespace lfm25
