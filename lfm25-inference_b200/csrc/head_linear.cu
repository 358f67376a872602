// One small matrix product per attention head: moving a head's up-projection to the other side of an attention over
// latents (query times key projection before it, weighted latent times value projection after it).
#include "launch.h"
#include "stack_common.cuh"

namespace lfm25 {

namespace {

template <typename T>
struct HeadLinearArgs {
    const T* x;
    size_t x_pitch, x_head;
    const __nv_bfloat16* weight;
    size_t w_head, w_n, w_k;
    T* y;
    size_t y_pitch;
    const T* gate;
    size_t gate_pitch;
    uint32_t tokens, n, k, heads;
    uint32_t column_tiles;
};

// ------------------------------------------------------------------------------------------------ tensor cores, bf16

constexpr uint32_t kThreads = 128;
constexpr uint32_t kRows = 64;        // tokens per CTA, 16 per warp
constexpr uint32_t kDepth = 64;       // inputs per round
constexpr uint32_t kPad = 8;          // elements behind each row of shared memory: conflict-free ldmatrix

constexpr uint32_t kStages = 4;       // rounds in shared memory, one of them being multiplied

template <uint32_t COLUMNS, bool OUTPUT_MAJOR>
struct Tile {
    __nv_bfloat16 x[kRows][kDepth + kPad];
    __nv_bfloat16 w[OUTPUT_MAJOR ? COLUMNS : kDepth][(OUTPUT_MAJOR ? kDepth : COLUMNS) + kPad];
};

// COLUMNS outputs per CTA.  OUTPUT_MAJOR: the weight's inputs are contiguous (w_k == 1), else its outputs are (w_n == 1).
template <uint32_t COLUMNS, bool OUTPUT_MAJOR>
__global__ void __launch_bounds__(kThreads)
head_linear_mma_kernel(const HeadLinearArgs<__nv_bfloat16> args) {
    extern __shared__ __align__(16) unsigned char head_linear_smem[];
    Tile<COLUMNS, OUTPUT_MAJOR>* tiles = reinterpret_cast<Tile<COLUMNS, OUTPUT_MAJOR>*>(head_linear_smem);
    pdl_launch_dependents();
    const uint32_t tile = blockIdx.x % args.column_tiles;
    const uint32_t head = blockIdx.x / args.column_tiles % args.heads;
    const uint32_t row0 = blockIdx.x / args.column_tiles / args.heads * kRows;
    const uint32_t column0 = tile * COLUMNS;
    const __nv_bfloat16* x = args.x + head * args.x_head;
    const __nv_bfloat16* weight = args.weight + head * args.w_head;
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t rounds = (args.k + kDepth - 1) / kDepth;
    auto load_weight = [&](uint32_t round) {
        auto& target = tiles[round % kStages].w;
#pragma unroll
        for (uint32_t part = 0; part < COLUMNS * kDepth / 8 / kThreads; ++part) {
            const uint32_t item = threadIdx.x + part * kThreads;
            constexpr uint32_t kPerRow = (OUTPUT_MAJOR ? kDepth : COLUMNS) / 8;
            const uint32_t outer = item / kPerRow, inner = item % kPerRow * 8;
            const uint32_t n = column0 + (OUTPUT_MAJOR ? outer : inner);
            const uint32_t k = round * kDepth + (OUTPUT_MAJOR ? inner : outer);
            const bool inside = n < args.n && k < args.k;
            copy_async_16(&target[outer][inner], weight + (inside ? n * args.w_n + k * args.w_k : 0), inside);
        }
    };
    auto load_input = [&](uint32_t round) {
        auto& target = tiles[round % kStages].x;
#pragma unroll
        for (uint32_t part = 0; part < kRows * kDepth / 8 / kThreads; ++part) {
            const uint32_t item = threadIdx.x + part * kThreads;
            const uint32_t row = item / (kDepth / 8), inner = item % (kDepth / 8) * 8;
            const bool inside = row0 + row < args.tokens && round * kDepth + inner < args.k;
            copy_async_16(&target[row][inner], x + (inside ? (row0 + row) * args.x_pitch + round * kDepth + inner : 0), inside);
        }
    };
    for (uint32_t round = 0; round < kStages - 1 && round < rounds; ++round) load_weight(round);
    pdl_wait();
    for (uint32_t round = 0; round < kStages - 1; ++round) {
        if (round < rounds) load_input(round);
        copy_async_commit();
    }
    float sum[COLUMNS / 8][4] = {};
    for (uint32_t round = 0; round < rounds; ++round) {
        copy_async_wait<kStages - 2>();
        __syncthreads();
        if (round + kStages - 1 < rounds) {
            load_weight(round + kStages - 1);
            load_input(round + kStages - 1);
        }
        copy_async_commit();
        const auto& x_tile = tiles[round % kStages].x;
        const auto& w_tile = tiles[round % kStages].w;
#pragma unroll
        for (uint32_t step = 0; step < kDepth / 16; ++step) {
            uint32_t a0, a1, a2, a3;
            ldmatrix_x4(smem_u32(&x_tile[warp * 16 + (lane & 15)][step * 16 + (lane >> 4) * 8]), a0, a1, a2, a3);
#pragma unroll
            for (uint32_t pair = 0; pair < COLUMNS / 16; ++pair) {
                uint32_t b0, b1, b2, b3;
                if constexpr (OUTPUT_MAJOR) {
                    ldmatrix_x4(smem_u32(&w_tile[pair * 16 + (lane >> 4) * 8 + (lane & 7)]
                                                [step * 16 + (lane >> 3 & 1) * 8]),
                                b0, b1, b2, b3);
                } else {
                    ldmatrix_x4_trans(smem_u32(&w_tile[step * 16 + (lane >> 3 & 1) * 8 + (lane & 7)]
                                                      [pair * 16 + (lane >> 4) * 8]),
                                      b0, b1, b2, b3);
                }
                mma_bf16_16816(sum[2 * pair], a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(sum[2 * pair + 1], a0, a1, a2, a3, b2, b3);
            }
        }
    }
#pragma unroll
    for (uint32_t part = 0; part < 2; ++part) {
        const uint32_t token = row0 + warp * 16 + (lane >> 2) + part * 8;
        if (token >= args.tokens) {
            continue;
        }
#pragma unroll
        for (uint32_t tile_column = 0; tile_column < COLUMNS / 8; ++tile_column) {
            const uint32_t column = column0 + tile_column * 8 + (lane & 3) * 2;
            if (column >= args.n) {
                continue;
            }
            float low = sum[tile_column][2 * part], high = sum[tile_column][2 * part + 1];
            const size_t at = static_cast<size_t>(head) * args.n + column;
            if (args.gate != nullptr) {
                const __nv_bfloat16* gate = args.gate + token * args.gate_pitch + at;
                low *= sigmoidf(__bfloat162float(gate[0]));
                high *= sigmoidf(__bfloat162float(gate[1]));
            }
            *reinterpret_cast<uint32_t*>(args.y + token * args.y_pitch + at) = pack_bf16x2(low, high);
        }
    }
}

// ------------------------------------------------------------------------------------------------ plain arithmetic

constexpr uint32_t kPlainThreads = 256;
constexpr uint32_t kTile = 64;
constexpr uint32_t kTileDepth = 16;

// 64 tokens x 64 outputs per CTA, 4 x 4 per thread, products and sums in f32: the f32 type and sizes without 16-byte rows
template <typename T>
__global__ void __launch_bounds__(kPlainThreads)
head_linear_plain_kernel(const HeadLinearArgs<T> args) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float x_tile[kTileDepth][kTile + 4];
    __shared__ float w_tile[kTileDepth][kTile + 4];
    const uint32_t column0 = blockIdx.x % args.column_tiles * kTile;
    const uint32_t head = blockIdx.x / args.column_tiles % args.heads;
    const uint32_t row0 = blockIdx.x / args.column_tiles / args.heads * kTile;
    const T* x = args.x + head * args.x_head;
    const __nv_bfloat16* weight = args.weight + head * args.w_head;
    const uint32_t tx = threadIdx.x & 15;
    const uint32_t ty = threadIdx.x >> 4;
    float sum[4][4] = {};
    for (uint32_t depth = 0; depth < args.k; depth += kTileDepth) {
#pragma unroll
        for (uint32_t part = 0; part < kTile * kTileDepth / kPlainThreads; ++part) {
            const uint32_t item = threadIdx.x + part * kPlainThreads;
            {
                const uint32_t row = row0 + item / kTileDepth, k = depth + item % kTileDepth;
                x_tile[item % kTileDepth][item / kTileDepth] =
                    row < args.tokens && k < args.k ? to_float<T>(x[row * args.x_pitch + k]) : 0.0f;
            }
            // neighbouring threads read along the weight's contiguous dimension
            const uint32_t inner = args.w_k == 1 ? item % kTileDepth : item / kTile;
            const uint32_t column = args.w_k == 1 ? item / kTileDepth : item % kTile;
            const uint32_t n = column0 + column, k = depth + inner;
            w_tile[inner][column] =
                n < args.n && k < args.k ? __bfloat162float(weight[n * args.w_n + k * args.w_k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (uint32_t inner = 0; inner < kTileDepth; ++inner) {
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
            const uint32_t token = row0 + ty * 4 + i, column = column0 + tx * 4 + j;
            if (token < args.tokens && column < args.n) {
                const size_t at = static_cast<size_t>(head) * args.n + column;
                float value = sum[i][j];
                if (args.gate != nullptr) value *= sigmoidf(to_float<T>(args.gate[token * args.gate_pitch + at]));
                args.y[token * args.y_pitch + at] = from_float<T>(value);
            }
        }
    }
}

template <typename T>
HeadLinearArgs<T> typed_args(const HeadLinearLaunch& launch) {
    HeadLinearArgs<T> args;
    args.x = static_cast<const T*>(launch.x);
    args.x_pitch = launch.x_pitch;
    args.x_head = launch.x_head;
    args.weight = static_cast<const __nv_bfloat16*>(launch.weight);
    args.w_head = launch.w_head;
    args.w_n = launch.w_n;
    args.w_k = launch.w_k;
    args.y = static_cast<T*>(launch.y);
    args.y_pitch = launch.y_pitch;
    args.gate = static_cast<const T*>(launch.gate);
    args.gate_pitch = launch.gate_pitch;
    args.tokens = static_cast<uint32_t>(launch.tokens);
    args.n = static_cast<uint32_t>(launch.n);
    args.k = static_cast<uint32_t>(launch.k);
    args.heads = launch.heads;
    args.column_tiles = 0;
    return args;
}

template <typename T>
cudaError_t launch_plain(cudaStream_t stream, const HeadLinearLaunch& launch) {
    HeadLinearArgs<T> args = typed_args<T>(launch);
    args.column_tiles = (args.n + kTile - 1) / kTile;
    const size_t blocks = static_cast<size_t>(args.column_tiles) * args.heads * ((args.tokens + kTile - 1) / kTile);
    return launch_kernel(head_linear_plain_kernel<T>, static_cast<unsigned int>(blocks), kPlainThreads, 0, stream, 1, args);
}

template <uint32_t COLUMNS>
cudaError_t launch_mma(cudaStream_t stream, const HeadLinearLaunch& launch) {
    HeadLinearArgs<__nv_bfloat16> args = typed_args<__nv_bfloat16>(launch);
    args.column_tiles = (args.n + COLUMNS - 1) / COLUMNS;
    const size_t blocks = static_cast<size_t>(args.column_tiles) * args.heads * ((args.tokens + kRows - 1) / kRows);
    const bool output_major = launch.w_k == 1;
    const auto kernel = output_major ? head_linear_mma_kernel<COLUMNS, true> : head_linear_mma_kernel<COLUMNS, false>;
    const size_t shared = kStages * (output_major ? sizeof(Tile<COLUMNS, true>) : sizeof(Tile<COLUMNS, false>));
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
    if (status != cudaSuccess) return status;
    return launch_kernel(kernel, static_cast<unsigned int>(blocks), kThreads, shared, stream, 1, args);
}

}  // namespace

cudaError_t launch_head_linear(cudaStream_t stream, const HeadLinearLaunch& launch) {
    if (launch.type == Activation::kF32) {
        return launch_plain<float>(stream, launch);
    }
    const size_t outer = launch.w_k == 1 ? launch.w_n : launch.w_k;
    const bool tensor = launch.n % 8 == 0 && launch.k % 8 == 0 && launch.x_pitch % 8 == 0 && launch.x_head % 8 == 0 &&
                        launch.w_head % 8 == 0 && outer % 8 == 0 && launch.y_pitch % 8 == 0 &&
                        aligned_to(launch.x, 16) && aligned_to(launch.weight, 16) && aligned_to(launch.y, 16);
    if (!tensor) {
        return launch_plain<__nv_bfloat16>(stream, launch);
    }
    // narrow tiles while the grid would not fill the machine
    const size_t wide = static_cast<size_t>(launch.heads) * ((launch.tokens + kRows - 1) / kRows) * ((launch.n + 63) / 64);
    return wide < 148 ? launch_mma<32>(stream, launch) : launch_mma<64>(stream, launch);
}

}  // namespace lfm25
