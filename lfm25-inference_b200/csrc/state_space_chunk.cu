// State-space recurrence over prompts as matrix products, for bf16 activations and states of up to 256 rows.
//
// With a_t = exp(-rate dt_t), A_t = a_1 ... a_t inside a chunk of 64 tokens and S the state before it,
//     y_t = A_t S^T C_t + sum_{s <= t} (A_t / A_s) dt_s (C_t . B_s) x_s + skip x_t
//     S  <- A_64 S + sum_s (A_64 / A_s) dt_s B_s x_s^T
// A CTA owns one segment, one head and 64 columns of its state, and walks the segment chunk by chunk: the state stays in
// f32 accumulators (its product B^T x is added there), C B^T and C S share the loads of C.  x, B and C are bf16 already;
// everything that the recurrence multiplies them with -- the decays, the triangle of weights, the state itself -- enters
// the tensor core as a sum of two bf16 values (16 significant bits).  The logarithms of the A_t are summed in double and
// kept as two floats, so that the ratio of two neighbours behind a long decay is exact.
#include <algorithm>

#include "launch.h"
#include "state_space.h"

namespace lfm25 {

namespace {

constexpr uint32_t kThreads = 256;
constexpr uint32_t kTokens = 64;
constexpr uint32_t kColumns = 64;
constexpr uint32_t kPad = 8;                            // elements behind each row: conflict-free ldmatrix
constexpr uint32_t kColumnPitch = kColumns + kPad;
constexpr size_t kSharedLimit = 227 * 1024;

struct Tables {
    float log_high[kTokens], log_low[kTokens];          // log2 A_t
    float step[kTokens];
    float into_state[kTokens];                          // (A_64 / A_s) dt_s
};

// Bytes of one buffer of a chunk's B, C and x
__host__ __device__ constexpr size_t chunk_bytes(uint32_t padded) {
    return (2 * kTokens * (padded + kPad) + kTokens * kColumnPitch) * 2;
}
constexpr size_t shared_bytes(uint32_t padded, uint32_t buffers) {
    // state and weighted x, both as two bf16 parts
    return buffers * chunk_bytes(padded) + 2 * (padded + kTokens) * kColumnPitch * 2 + sizeof(Tables);
}

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& high, uint32_t& low) {
    high = pack_bf16x2(a, b);
    const float2 rounded = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high));
    low = pack_bf16x2(a - rounded.x, b - rounded.y);
}

// UNITS: pieces of 16 state rows x 32 columns per warp (8 warps)
template <int UNITS>
__global__ void __launch_bounds__(kThreads, UNITS <= 2 ? 2 : 1)
state_space_chunk_kernel(const StateSpaceArgs<__nv_bfloat16> args, uint32_t column_blocks, uint32_t padded,
                         uint32_t buffers) {
    extern __shared__ __align__(16) unsigned char chunk_smem[];
    const uint32_t pitch = padded + kPad;
    __nv_bfloat16* tiles = reinterpret_cast<__nv_bfloat16*>(chunk_smem);
    const uint32_t tile_elements = static_cast<uint32_t>(chunk_bytes(padded) / 2);
    __nv_bfloat16* state_high = tiles + buffers * tile_elements;        // [padded][columns]
    __nv_bfloat16* state_low = state_high + padded * kColumnPitch;
    __nv_bfloat16* input_high = state_low + padded * kColumnPitch;      // [tokens][columns]
    __nv_bfloat16* input_low = input_high + kTokens * kColumnPitch;
    Tables& tables = *reinterpret_cast<Tables*>(input_low + kTokens * kColumnPitch);
    pdl_launch_dependents();
    pdl_wait();

    const uint32_t block = blockIdx.x % column_blocks;
    const uint32_t head = blockIdx.x / column_blocks % args.heads;
    const uint32_t segment = blockIdx.x / column_blocks / args.heads;
    const size_t slot = args.segments.slots[segment];
    if (slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t begin = args.segments.offsets[segment];
    const uint32_t stop = args.segments.offsets[segment + 1];
    const uint32_t end = stop < args.segments.num_tokens ? stop : static_cast<uint32_t>(args.segments.num_tokens);
    const uint32_t group = head / (args.heads / args.groups);
    const size_t inner = static_cast<size_t>(args.heads) * args.vdim;
    const uint32_t column0 = block * kColumns;
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t row0 = lane >> 2;
    const uint32_t pair = (lane & 3) * 2;
    const float rate_log2 = -state_rate(args, head) * kLog2e;
    const float skip = __bfloat162float(args.skip[head]);

    auto load_chunk = [&](uint32_t first, uint32_t buffer) {
        __nv_bfloat16* b = tiles + buffer * tile_elements;
        __nv_bfloat16* c = b + kTokens * pitch;
        __nv_bfloat16* x = c + kTokens * pitch;
        const uint32_t vectors = padded / 8;
        for (uint32_t item = threadIdx.x; item < kTokens * vectors; item += kThreads) {
            const uint32_t row = item / vectors, n = item % vectors * 8;
            const bool inside = first + row < end && n < args.size;
            const __nv_bfloat16* source = args.mixed;
            if (inside) source += static_cast<size_t>(first + row) * args.mixed_pitch + inner + group * args.size + n;
            copy_async_16(b + row * pitch + n, source, inside);
            copy_async_16(c + row * pitch + n, source + (inside ? args.groups * args.size : 0), inside);
        }
        for (uint32_t item = threadIdx.x; item < kTokens * kColumns / 8; item += kThreads) {
            const uint32_t row = item / (kColumns / 8), v = item % (kColumns / 8) * 8;
            const bool inside = first + row < end && column0 + v < args.vdim;
            copy_async_16(x + row * kColumnPitch + v,
                       args.mixed + (inside ? static_cast<size_t>(first + row) * args.mixed_pitch + head * args.vdim +
                                                  column0 + v
                                            : 0),
                       inside);
        }
        copy_async_commit();
    };
    // warp 0: step sizes of a chunk, two tokens per lane
    auto load_steps = [&](uint32_t first, float (&steps)[2]) {
#pragma unroll
        for (uint32_t i = 0; i < 2; ++i) {
            const uint32_t token = first + 2 * lane + i;
            steps[i] = token < end ? step_size(args, token, head) : 0.0f;
        }
    };

    float* state = state_of(args, slot, head);
    float held[UNITS][4][4];
#pragma unroll
    for (int unit = 0; unit < UNITS; ++unit) {
        const uint32_t piece = warp + 8 * unit;
        const uint32_t n = piece / 2 * 16 + row0;
#pragma unroll
        for (uint32_t tile = 0; tile < 4; ++tile) {
            const uint32_t v = column0 + piece % 2 * 32 + tile * 8 + pair;
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                float2 value = make_float2(0.0f, 0.0f);
                if (n + half * 8 < args.size && v < args.vdim) {
                    value = *reinterpret_cast<const float2*>(state + static_cast<size_t>(n + half * 8) * args.vdim + v);
                }
                held[unit][tile][2 * half] = value.x;
                held[unit][tile][2 * half + 1] = value.y;
            }
        }
    }
    float steps[2] = {};
    load_chunk(begin, 0);
    if (warp == 0) load_steps(begin, steps);
    uint32_t buffer = 0;
    for (uint32_t first = begin; first < end; first += kTokens) {
        if (warp == 0) {
            // log2 A_t: scan over the chunk in double
            const double low = static_cast<double>(rate_log2 * steps[0]);
            const double both = low + static_cast<double>(rate_log2 * steps[1]);
            double inclusive = both;
#pragma unroll
            for (uint32_t delta = 1; delta < 32; delta <<= 1) {
                const double other = __shfl_up_sync(0xffffffffu, inclusive, delta);
                inclusive += lane >= delta ? other : 0.0;
            }
            const double total = __shfl_sync(0xffffffffu, inclusive, 31);
            const double logs[2] = {inclusive - both + low, inclusive};
#pragma unroll
            for (uint32_t i = 0; i < 2; ++i) {
                const uint32_t t = 2 * lane + i;
                const float high = static_cast<float>(logs[i]);
                tables.log_high[t] = high;
                tables.log_low[t] = static_cast<float>(logs[i] - static_cast<double>(high));
                tables.step[t] = steps[i];
                tables.into_state[t] = fast_exp2(static_cast<float>(total - logs[i])) * steps[i];
            }
            if (first + kTokens < end) load_steps(first + kTokens, steps);
        }
        copy_async_wait<0>();
        __syncthreads();
        if (buffers == 2 && first + kTokens < end) load_chunk(first + kTokens, buffer ^ 1);
        const __nv_bfloat16* b = tiles + buffer * tile_elements;
        const __nv_bfloat16* c = b + kTokens * pitch;
        const __nv_bfloat16* x = c + kTokens * pitch;
        // ---- the state and the weighted inputs as two bf16 parts each
#pragma unroll
        for (int unit = 0; unit < UNITS; ++unit) {
            const uint32_t piece = warp + 8 * unit;
            if (piece / 2 * 16 < padded) {
#pragma unroll
                for (uint32_t tile = 0; tile < 4; ++tile) {
#pragma unroll
                    for (uint32_t half = 0; half < 2; ++half) {
                        uint32_t high, low;
                        split_pair(held[unit][tile][2 * half], held[unit][tile][2 * half + 1], high, low);
                        const uint32_t row = piece / 2 * 16 + row0 + half * 8;
                        const uint32_t at = row * kColumnPitch + piece % 2 * 32 + tile * 8 + pair;
                        *reinterpret_cast<uint32_t*>(state_high + at) = high;
                        *reinterpret_cast<uint32_t*>(state_low + at) = low;
                    }
                }
            }
        }
#pragma unroll
        for (uint32_t item = threadIdx.x; item < kTokens * kColumns / 8; item += kThreads) {
            const uint32_t row = item / (kColumns / 8), v = item % (kColumns / 8) * 8;
            float value[8];
            load_values<8>(x + row * kColumnPitch + v, value);
            const float weight = tables.into_state[row];
            uint32_t high[4], low[4];
#pragma unroll
            for (uint32_t i = 0; i < 4; ++i) split_pair(value[2 * i] * weight, value[2 * i + 1] * weight, high[i], low[i]);
            *reinterpret_cast<uint4*>(input_high + row * kColumnPitch + v) = make_uint4(high[0], high[1], high[2], high[3]);
            *reinterpret_cast<uint4*>(input_low + row * kColumnPitch + v) = make_uint4(low[0], low[1], low[2], low[3]);
        }
        __syncthreads();

        // ---- outputs: 16 tokens x 32 columns per warp
        {
            const uint32_t tile_row = warp & 3;
            const uint32_t half_column = (warp >> 2) * 32;
            float products[8][4] = {}, carried[4][4] = {};
            for (uint32_t k = 0; k < padded; k += 16) {
                uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
                ldmatrix_x4(smem_u32(c + (tile_row * 16 + (lane & 15)) * pitch + k + (lane >> 4) * 8), a0, a1, a2, a3);
#pragma unroll
                for (uint32_t j = 0; j < 4; ++j) {
                    if (j <= tile_row) {
                        ldmatrix_x4(smem_u32(b + (j * 16 + (lane >> 4) * 8 + (lane & 7)) * pitch + k + (lane >> 3 & 1) * 8),
                                    b0, b1, b2, b3);
                        mma_bf16_16816(products[2 * j], a0, a1, a2, a3, b0, b1);
                        mma_bf16_16816(products[2 * j + 1], a0, a1, a2, a3, b2, b3);
                    }
                }
#pragma unroll
                for (uint32_t q = 0; q < 2; ++q) {
                    const uint32_t at = (k + (lane >> 3 & 1) * 8 + (lane & 7)) * kColumnPitch + half_column + q * 16 +
                                        (lane >> 4) * 8;
                    ldmatrix_x4_trans(smem_u32(state_high + at), b0, b1, b2, b3);
                    mma_bf16_16816(carried[2 * q], a0, a1, a2, a3, b0, b1);
                    mma_bf16_16816(carried[2 * q + 1], a0, a1, a2, a3, b2, b3);
                    ldmatrix_x4_trans(smem_u32(state_low + at), b0, b1, b2, b3);
                    mma_bf16_16816(carried[2 * q], a0, a1, a2, a3, b0, b1);
                    mma_bf16_16816(carried[2 * q + 1], a0, a1, a2, a3, b2, b3);
                }
            }
            const uint32_t t[2] = {tile_row * 16 + row0, tile_row * 16 + row0 + 8};
            const float log_high[2] = {tables.log_high[t[0]], tables.log_high[t[1]]};
            const float log_low[2] = {tables.log_low[t[0]], tables.log_low[t[1]]};
            float sum[4][4] = {};
#pragma unroll
            for (uint32_t j = 0; j < 4; ++j) {
                if (j > tile_row) {
                    continue;
                }
                uint32_t high[4], low[4];
#pragma unroll
                for (uint32_t part = 0; part < 2; ++part) {            // 8 tokens s each
                    const uint32_t s = j * 16 + part * 8 + pair;
                    const float2 s_high = *reinterpret_cast<const float2*>(tables.log_high + s);
                    const float2 s_low = *reinterpret_cast<const float2*>(tables.log_low + s);
                    const float2 s_step = *reinterpret_cast<const float2*>(tables.step + s);
#pragma unroll
                    for (uint32_t half = 0; half < 2; ++half) {
                        const float first_weight =
                            fast_exp2((log_high[half] - s_high.x) + (log_low[half] - s_low.x)) * s_step.x;
                        const float second_weight =
                            fast_exp2((log_high[half] - s_high.y) + (log_low[half] - s_low.y)) * s_step.y;
                        const float first_value = s <= t[half] ? products[2 * j + part][2 * half] * first_weight : 0.0f;
                        const float second_value =
                            s + 1 <= t[half] ? products[2 * j + part][2 * half + 1] * second_weight : 0.0f;
                        split_pair(first_value, second_value, high[2 * part + half], low[2 * part + half]);
                    }
                }
#pragma unroll
                for (uint32_t q = 0; q < 2; ++q) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(smem_u32(x + (j * 16 + (lane >> 3 & 1) * 8 + (lane & 7)) * kColumnPitch + half_column +
                                               q * 16 + (lane >> 4) * 8),
                                      b0, b1, b2, b3);
                    mma_bf16_16816(sum[2 * q], high[0], high[1], high[2], high[3], b0, b1);
                    mma_bf16_16816(sum[2 * q + 1], high[0], high[1], high[2], high[3], b2, b3);
                    mma_bf16_16816(sum[2 * q], low[0], low[1], low[2], low[3], b0, b1);
                    mma_bf16_16816(sum[2 * q + 1], low[0], low[1], low[2], low[3], b2, b3);
                }
            }
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                const uint32_t token = first + t[half];
                const float carry = fast_exp2(log_high[half] + log_low[half]);
                if (token < end) {
#pragma unroll
                    for (uint32_t tile = 0; tile < 4; ++tile) {
                        const uint32_t local = half_column + tile * 8 + pair;
                        if (column0 + local < args.vdim) {
                            const float2 input = __bfloat1622float2(
                                *reinterpret_cast<const __nv_bfloat162*>(x + t[half] * kColumnPitch + local));
                            const float low = fmaf(skip, input.x, fmaf(carry, carried[tile][2 * half], sum[tile][2 * half]));
                            const float high =
                                fmaf(skip, input.y, fmaf(carry, carried[tile][2 * half + 1], sum[tile][2 * half + 1]));
                            *reinterpret_cast<uint32_t*>(args.out + token * inner + head * args.vdim + column0 + local) =
                                pack_bf16x2(low, high);
                        }
                    }
                }
            }
        }

        // ---- the state behind the chunk
        const float decay = fast_exp2(tables.log_high[kTokens - 1] + tables.log_low[kTokens - 1]);
#pragma unroll
        for (int unit = 0; unit < UNITS; ++unit) {
            const uint32_t piece = warp + 8 * unit;
            const uint32_t n0 = piece / 2 * 16;
            if (n0 >= padded) {
                continue;
            }
#pragma unroll
            for (uint32_t tile = 0; tile < 4; ++tile) {
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) held[unit][tile][i] *= decay;
            }
#pragma unroll
            for (uint32_t k = 0; k < kTokens; k += 16) {
                uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
                ldmatrix_x4_trans(smem_u32(b + (k + (lane >> 4) * 8 + (lane & 7)) * pitch + n0 + (lane >> 3 & 1) * 8), a0, a1,
                                  a2, a3);
#pragma unroll
                for (uint32_t q = 0; q < 2; ++q) {
                    const uint32_t at = (k + (lane >> 3 & 1) * 8 + (lane & 7)) * kColumnPitch + piece % 2 * 32 + q * 16 +
                                        (lane >> 4) * 8;
                    ldmatrix_x4_trans(smem_u32(input_high + at), b0, b1, b2, b3);
                    mma_bf16_16816(held[unit][2 * q], a0, a1, a2, a3, b0, b1);
                    mma_bf16_16816(held[unit][2 * q + 1], a0, a1, a2, a3, b2, b3);
                    ldmatrix_x4_trans(smem_u32(input_low + at), b0, b1, b2, b3);
                    mma_bf16_16816(held[unit][2 * q], a0, a1, a2, a3, b0, b1);
                    mma_bf16_16816(held[unit][2 * q + 1], a0, a1, a2, a3, b2, b3);
                }
            }
        }
        __syncthreads();
        if (buffers == 2) {
            buffer ^= 1;
        } else if (first + kTokens < end) {
            load_chunk(first + kTokens, 0);
        }
    }
#pragma unroll
    for (int unit = 0; unit < UNITS; ++unit) {
        const uint32_t piece = warp + 8 * unit;
        const uint32_t n = piece / 2 * 16 + row0;
#pragma unroll
        for (uint32_t tile = 0; tile < 4; ++tile) {
            const uint32_t v = column0 + piece % 2 * 32 + tile * 8 + pair;
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                if (n + half * 8 < args.size && v < args.vdim) {
                    *reinterpret_cast<float2*>(state + static_cast<size_t>(n + half * 8) * args.vdim + v) =
                        make_float2(held[unit][tile][2 * half], held[unit][tile][2 * half + 1]);
                }
            }
        }
    }
}

}  // namespace

bool state_space_chunk_supports(const StateSpaceLaunch& launch) {
    return launch.type == Activation::kBf16 && launch.segments.offsets != nullptr && launch.size % 8 == 0 &&
           launch.size <= 256 && launch.vdim % 8 == 0 && launch.mixed_pitch % 8 == 0 && aligned_to(launch.mixed, 16) &&
           aligned_to(launch.out, 4) && launch.record.offset % 16 == 0 && launch.record.stride % 16 == 0 &&
           aligned_to(launch.record.base, 16);
}

cudaError_t launch_state_space_chunk(cudaStream_t stream, const StateSpaceLaunch& launch) {
    const uint32_t padded = (launch.size + 15) / 16 * 16;
    const uint32_t column_blocks = (launch.vdim + kColumns - 1) / kColumns;
    const size_t blocks = launch.segments.num_segments * launch.heads * column_blocks;
    // two CTAs per SM hide each other's loads; where there are not enough of them, a second buffer does
    const bool alone = blocks <= 148 || shared_bytes(padded, 1) > kSharedLimit / 2 - 1024;
    const uint32_t buffers = alone && shared_bytes(padded, 2) <= kSharedLimit ? 2 : 1;
    const size_t shared = shared_bytes(padded, buffers);
    const auto kernel = padded <= 64    ? state_space_chunk_kernel<1>
                        : padded <= 128 ? state_space_chunk_kernel<2>
                                        : state_space_chunk_kernel<4>;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
    if (status != cudaSuccess) return status;
    return launch_kernel(kernel, static_cast<unsigned int>(blocks), kThreads, shared, stream, 1,
                         state_space_args<__nv_bfloat16>(launch), column_blocks, padded, buffers);
}

}  // namespace lfm25
