// Decode attention of the layer stack for bf16 activations: one query token per sequence, any grouping of up to 16
// query heads per key/value head, query/key and value sizes up to 256, an optional chunk mask.
//
// One CTA per token, key/value head and split of the visible pages; its four warps take pages in turn, each through a
// ring of its own that TMA fills (one box of 64 dimensions x 16 keys per copy, 128-byte swizzle).  A page is 16 keys of
// one head: S = Q K^T and O += P V are mma.sync tiles whose 16 rows are the query heads of the group.  The weights enter
// the second product as a sum of two bf16 values (16 significant bits); maximum, sum and accumulators are f32.  The four
// warps merge through shared memory, the splits of a token through the distributed shared memory of their cluster.
#include <cooperative_groups.h>
#include <math.h>

#include <algorithm>

#include "launch.h"
#include "options.h"
#include "stack_attention.h"
#include "stack_common.cuh"

namespace lfm25 {

namespace {

namespace cg = cooperative_groups;

constexpr uint32_t kWarps = 4;
constexpr uint32_t kThreads = kWarps * 32;
constexpr uint32_t kBoxBytes = kPageSize * 128;   // 16 keys x 64 dimensions
constexpr uint32_t kGroupRows = 16;

template <uint32_t KC, uint32_t VC>
struct Layout {
    static constexpr uint32_t kStageBytes = (KC + VC) * kBoxBytes;
    static constexpr uint32_t kStages = KC + VC <= 2 ? 4 : (KC + VC <= 4 ? 3 : 2);
    static constexpr uint32_t kRingBytes = kWarps * kStages * kStageBytes;
    static constexpr uint32_t kColumns = 64 * VC;
    // the warps' partial results reuse the ring once every page has been consumed
    static constexpr uint32_t kPartialBytes = kWarps * kGroupRows * kColumns * 4;
    static constexpr uint32_t kBodyBytes = kRingBytes > kPartialBytes ? kRingBytes : kPartialBytes;
    // behind it: the CTA's result, maxima and sums per warp, maxima and sums per CTA, barriers, abort flag
    static constexpr uint32_t kResultBytes = kGroupRows * kColumns * 4;
    static constexpr uint32_t kSharedBytes = kBodyBytes + kResultBytes + (kWarps + 1) * kGroupRows * 8 +
                                             kWarps * kStages * 8 + 16 + 1024;
    static_assert(kSharedBytes <= 227 * 1024, "shared memory");
};

struct Params {
    StackAttentionShape shape;
    const __nv_bfloat16* query;
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* request_slots;
    const uint32_t* positions;
    __nv_bfloat16* out;
    size_t out_pitch;
    unsigned int* status;
    uint32_t splits;
    uint64_t wait_limit;
};

template <uint32_t KC, uint32_t VC>
__global__ void __launch_bounds__(kThreads)
stack_attention_decode_kernel(const __grid_constant__ CUtensorMap key_map, const __grid_constant__ CUtensorMap value_map,
                              const Params p) {
    using L = Layout<KC, VC>;
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    extern __shared__ uint8_t decode_smem[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(decode_smem) + 1023) & ~uintptr_t(1023));
    float* partial = reinterpret_cast<float*>(smem);                                  // [warp][row][column]
    float* result = reinterpret_cast<float*>(smem + L::kBodyBytes);                   // [row][column]
    float* warp_top = result + kGroupRows * L::kColumns;                              // [warp][row]
    float* warp_sums = warp_top + kWarps * kGroupRows;
    float* cta_top = warp_sums + kWarps * kGroupRows;                                 // [row]
    float* cta_sum = cta_top + kGroupRows;
    uint8_t* barriers = reinterpret_cast<uint8_t*>(cta_sum + kGroupRows);
    volatile uint32_t* abort_flag = reinterpret_cast<volatile uint32_t*>(barriers + kWarps * L::kStages * 8);
    const uint32_t ring = smem_u32(smem) + warp * L::kStages * L::kStageBytes;
    const uint32_t bar = smem_u32(barriers) + warp * L::kStages * 8;
    pdl_launch_dependents();
    if (threadIdx.x == 0) *abort_flag = 0;
    if (lane == 0) {
        tma_prefetch_descriptor(&key_map);
        tma_prefetch_descriptor(&value_map);
        for (uint32_t stage = 0; stage < L::kStages; ++stage) mbar_init(bar + 8 * stage, 1);
        fence_barrier_init();
    }
    __syncthreads();
    pdl_wait();

    const uint32_t split = blockIdx.x % p.splits;
    const uint32_t kv_head = blockIdx.x / p.splits % p.shape.kv_heads;
    const size_t token = blockIdx.x / p.splits / p.shape.kv_heads;
    const uint32_t group = p.shape.heads / p.shape.kv_heads;
    const size_t table_row = p.request_slots[token];
    const uint32_t position = p.positions[token];
    const uint32_t first = first_visible(position, p.shape.chunk);
    const bool valid = table_row < p.block_table_rows && position / kPageSize < p.block_table_stride;
    const uint32_t first_page = first / kPageSize;
    const uint32_t pages = valid ? position / kPageSize - first_page + 1 : 0;
    const uint32_t* table = p.block_tables + (valid ? table_row * p.block_table_stride : 0);
    // this warp's pages: first_page + mine, + stride, ...
    const uint32_t stride = kWarps * p.splits;
    const uint32_t mine = split * kWarps + warp;
    const uint32_t count = pages > mine ? (pages - mine + stride - 1) / stride : 0;

    // entry of this warp's page `index`; read 32 at a time
    uint32_t held = 0;
    uint32_t held_base = 0xffffffffu;
    auto entry_of = [&](uint32_t index) -> uint32_t {
        const uint32_t base = index & ~31u;
        if (base != held_base) {
            held_base = base;
            held = base + lane < count ? __ldg(table + first_page + mine + (base + lane) * stride) : 0xffffffffu;
        }
        return __shfl_sync(0xffffffffu, held, index & 31);
    };
    uint32_t usable = 0;        // bit per stage: the page in it exists
    auto issue = [&](uint32_t index) {
        const uint32_t stage = index % L::kStages;
        const uint32_t entry = entry_of(index);
        const bool exists = entry < p.num_pages;
        usable = exists ? usable | (1u << stage) : usable & ~(1u << stage);
        if (lane == 0) {
            // a page that does not exist is read as page 0 and not used
            const int32_t row = static_cast<int32_t>(((exists ? entry : 0) * p.shape.kv_heads + kv_head) * kPageSize);
            const uint32_t target = ring + stage * L::kStageBytes;
            mbar_arrive_expect_tx(bar + 8 * stage, L::kStageBytes);
#pragma unroll
            for (uint32_t chunk = 0; chunk < KC; ++chunk) {
                tma_load_2d(target + chunk * kBoxBytes, &key_map, bar + 8 * stage, static_cast<int32_t>(chunk * 64), row);
            }
#pragma unroll
            for (uint32_t chunk = 0; chunk < VC; ++chunk) {
                tma_load_2d(target + (KC + chunk) * kBoxBytes, &value_map, bar + 8 * stage,
                            static_cast<int32_t>(chunk * 64), row);
            }
        }
    };
    uint32_t issued = 0;
    for (; issued < L::kStages && issued < count; ++issued) issue(issued);

    // query fragments: row = head of the group, times nothing (the scale is applied to the f32 scores)
    const uint32_t row0 = lane >> 2;
    const uint32_t pair = (lane & 3) * 2;
    uint32_t query[KC * 4][4];
    const __nv_bfloat16* query_rows = p.query + (token * p.shape.heads + static_cast<size_t>(kv_head) * group) * p.shape.dim;
#pragma unroll
    for (uint32_t ks = 0; ks < KC * 4; ++ks) {
#pragma unroll
        for (uint32_t part = 0; part < 4; ++part) {
            const uint32_t row = row0 + (part & 1) * 8;
            const uint32_t dim = ks * 16 + pair + (part >> 1) * 8;
            query[ks][part] = row < group && dim < p.shape.dim
                                  ? *reinterpret_cast<const uint32_t*>(query_rows + row * p.shape.dim + dim)
                                  : 0u;
        }
    }

    float out[VC * 8][4];
#pragma unroll
    for (uint32_t n = 0; n < VC * 8; ++n) {
#pragma unroll
        for (uint32_t i = 0; i < 4; ++i) out[n][i] = 0.0f;
    }
    float top[2] = {-INFINITY, -INFINITY};
    float sum[2] = {0.0f, 0.0f};
    const float scale_log2 = p.shape.scale * kLog2e;
    bool ok = true;
    uint32_t waited = 0;
    for (uint32_t index = 0; index < count; ++index) {
        const uint32_t stage = index % L::kStages;
        if (!__all_sync(0xffffffffu, mbar_wait_bounded(bar + 8 * stage, (index / L::kStages) & 1, p.wait_limit))) {
            ok = false;
            break;
        }
        waited = index + 1;
        const uint32_t key_base = ring + stage * L::kStageBytes;
        const uint32_t value_base = key_base + KC * kBoxBytes;
        const uint32_t page_first = (first_page + mine + index * stride) * kPageSize;
        if (usable >> stage & 1u) {
            float scores[2][4] = {};
#pragma unroll
            for (uint32_t ks = 0; ks < KC * 4; ++ks) {
                const uint32_t key = (lane >> 4) * 8 + (lane & 7);
                const uint32_t part = (ks & 3) * 2 + (lane >> 3 & 1);
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(key_base + (ks >> 2) * kBoxBytes + key * 128 + ((part ^ (key & 7)) << 4), b0, b1, b2, b3);
                mma_bf16_16816(scores[0], query[ks][0], query[ks][1], query[ks][2], query[ks][3], b0, b1);
                mma_bf16_16816(scores[1], query[ks][0], query[ks][1], query[ks][2], query[ks][3], b2, b3);
            }
            const bool whole = page_first >= first && page_first + kPageSize - 1 <= position;
            if (!whole) {
                if (page_first + kPageSize - 1 > position) {
                    // value rows behind the last key may hold anything, and zero times a NaN pattern is NaN
                    for (uint32_t item = lane; item < VC * kPageSize * 8; item += 32) {
                        const uint32_t key = item / 8 % kPageSize;
                        if (page_first + key > position) {
                            asm volatile("st.shared.v4.u32 [%0], {%1, %1, %1, %1};" ::"r"(
                                             value_base + item / (kPageSize * 8) * kBoxBytes + key * 128 + item % 8 * 16),
                                         "r"(0u)
                                         : "memory");
                        }
                    }
                    __syncwarp();
                }
#pragma unroll
                for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {
                        const uint32_t key = page_first + n * 8 + pair + (i & 1);
                        if (key < first || key > position) scores[n][i] = -INFINITY;
                    }
                }
            }
            float rescale[2];
#pragma unroll
            for (uint32_t r = 0; r < 2; ++r) {
                float best = fmaxf(fmaxf(scores[0][2 * r], scores[0][2 * r + 1]),
                                   fmaxf(scores[1][2 * r], scores[1][2 * r + 1]));
                best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 1));
                best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 2));
                const float now = fmaxf(top[r], best);
                const float base = now == -INFINITY ? 0.0f : now;
                rescale[r] = fast_exp2((top[r] - base) * scale_log2);
                const float offset = -base * scale_log2;
                float total = 0.0f;
#pragma unroll
                for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                    for (uint32_t i = 0; i < 2; ++i) {
                        const float weight = fast_exp2(fmaf(scores[n][2 * r + i], scale_log2, offset));
                        scores[n][2 * r + i] = weight;
                        total += weight;
                    }
                }
                sum[r] = fmaf(sum[r], rescale[r], total);
                top[r] = now;
            }
            if (!__all_sync(0xffffffffu, rescale[0] == 1.0f && rescale[1] == 1.0f)) {
#pragma unroll
                for (uint32_t n = 0; n < VC * 8; ++n) {
                    out[n][0] *= rescale[0];
                    out[n][1] *= rescale[0];
                    out[n][2] *= rescale[1];
                    out[n][3] *= rescale[1];
                }
            }
            uint32_t high[4], low[4];
#pragma unroll
            for (uint32_t part = 0; part < 4; ++part) {
                const float a = scores[part >> 1][(part & 1) * 2];
                const float b = scores[part >> 1][(part & 1) * 2 + 1];
                high[part] = pack_bf16x2(a, b);
                const float2 rounded = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high[part]));
                low[part] = pack_bf16x2(a - rounded.x, b - rounded.y);
            }
#pragma unroll
            for (uint32_t n = 0; n < VC * 4; ++n) {     // 16 value dimensions at a time
                const uint32_t key = (lane >> 3 & 1) * 8 + (lane & 7);
                const uint32_t part = (n & 3) * 2 + (lane >> 4);
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(value_base + (n >> 2) * kBoxBytes + key * 128 + ((part ^ (key & 7)) << 4), b0, b1, b2,
                                  b3);
                mma_bf16_16816(out[2 * n], high[0], high[1], high[2], high[3], b0, b1);
                mma_bf16_16816(out[2 * n + 1], high[0], high[1], high[2], high[3], b2, b3);
                mma_bf16_16816(out[2 * n], low[0], low[1], low[2], low[3], b0, b1);
                mma_bf16_16816(out[2 * n + 1], low[0], low[1], low[2], low[3], b2, b3);
            }
        }
        __syncwarp();
        if (issued < count) {
            issue(issued);
            ++issued;
        }
    }
    if (!ok) {
        if (lane == 0) {
            *abort_flag = 1;
            record_wait_timeout(p.status, kTagStackDecode, blockIdx.x);
        }
        for (uint32_t index = waited; index < issued; ++index) {      // copies still in flight, each for a bounded time
            mbar_wait_bounded(bar + 8 * (index % L::kStages), (index / L::kStages) & 1, p.wait_limit);
        }
    }

    // ---- warps of the CTA
#pragma unroll
    for (uint32_t r = 0; r < 2; ++r) {
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
    }
    __syncthreads();          // every ring is drained
#pragma unroll
    for (uint32_t r = 0; r < 2; ++r) {
        const uint32_t row = row0 + r * 8;
        if (row < group) {
            if ((lane & 3) == 0) {
                warp_top[warp * kGroupRows + row] = top[r];
                warp_sums[warp * kGroupRows + row] = sum[r];
            }
            float* target = partial + (warp * kGroupRows + row) * L::kColumns + pair;
#pragma unroll
            for (uint32_t n = 0; n < VC * 8; ++n) {
                *reinterpret_cast<float2*>(target + n * 8) = make_float2(out[n][2 * r], out[n][2 * r + 1]);
            }
        }
    }
    __syncthreads();
    const uint32_t vdim = p.shape.vdim;
    __nv_bfloat16* target = p.out + token * p.out_pitch + static_cast<size_t>(kv_head) * group * vdim;
    const bool aborted = *abort_flag != 0;
    for (uint32_t item = threadIdx.x; item < group * vdim; item += kThreads) {
        const uint32_t row = item / vdim;
        const uint32_t column = item - row * vdim;
        float best = -INFINITY;
#pragma unroll
        for (uint32_t w = 0; w < kWarps; ++w) best = fmaxf(best, warp_top[w * kGroupRows + row]);
        const float base = best == -INFINITY ? 0.0f : best;
        float total = 0.0f, value = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < kWarps; ++w) {
            const float factor = fast_exp2((warp_top[w * kGroupRows + row] - base) * scale_log2);
            total = fmaf(warp_sums[w * kGroupRows + row], factor, total);
            value = fmaf(partial[(w * kGroupRows + row) * L::kColumns + column], factor, value);
        }
        if (p.splits == 1) {
            if (!aborted) target[item] = __float2bfloat16_rn(total > 0.0f ? value / total : 0.0f);
        } else {
            result[row * L::kColumns + column] = value;
            if (column == 0) {
                cta_top[row] = best;
                cta_sum[row] = total;
            }
        }
    }
    if (p.splits == 1) {
        return;
    }
    // ---- splits of the token: every CTA of the cluster finishes a share of the outputs
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    bool any_abort = false;
    for (uint32_t rank = 0; rank < p.splits; ++rank) {
        any_abort = any_abort || *cluster.map_shared_rank(const_cast<uint32_t*>(abort_flag), rank) != 0;
    }
    for (uint32_t item = threadIdx.x * p.splits + split; item < group * vdim; item += kThreads * p.splits) {
        const uint32_t row = item / vdim;
        const uint32_t column = item - row * vdim;
        float best = -INFINITY;
        for (uint32_t rank = 0; rank < p.splits; ++rank) {
            best = fmaxf(best, cluster.map_shared_rank(cta_top, rank)[row]);
        }
        const float base = best == -INFINITY ? 0.0f : best;
        float total = 0.0f, value = 0.0f;
        for (uint32_t rank = 0; rank < p.splits; ++rank) {
            const float factor = fast_exp2((cluster.map_shared_rank(cta_top, rank)[row] - base) * scale_log2);
            total = fmaf(cluster.map_shared_rank(cta_sum, rank)[row], factor, total);
            value = fmaf(cluster.map_shared_rank(result, rank)[row * L::kColumns + column], factor, value);
        }
        if (!any_abort) target[item] = __float2bfloat16_rn(total > 0.0f ? value / total : 0.0f);
    }
    cluster.sync();           // nobody leaves while its results are being read
}

template <uint32_t KC, uint32_t VC>
cudaError_t launch_sized(cudaStream_t stream, const StackAttentionLaunch& launch, uint32_t splits) {
    using L = Layout<KC, VC>;
    CUtensorMap key_map, value_map;
    if (!make_page_map(&key_map, launch, false) || !make_page_map(&value_map, launch, true)) {
        return cudaErrorInvalidValue;
    }
    const auto kernel = stack_attention_decode_kernel<KC, VC>;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                    static_cast<int>(L::kSharedBytes));
    if (status != cudaSuccess) return status;
    Params params;
    params.shape = launch.shape;
    params.query = static_cast<const __nv_bfloat16*>(launch.query);
    params.block_tables = launch.block_tables;
    params.block_table_stride = launch.block_table_stride;
    params.block_table_rows = launch.block_table_rows;
    params.num_pages = launch.num_pages;
    params.request_slots = launch.request_slots;
    params.positions = launch.positions;
    params.out = static_cast<__nv_bfloat16*>(launch.out);
    params.out_pitch = launch.out_pitch;
    params.status = launch.status;
    params.splits = splits;
    params.wait_limit = wait_limit_ns();
    const size_t blocks = launch.decode_tokens * launch.shape.kv_heads * splits;
    return launch_kernel(kernel, static_cast<unsigned int>(blocks), kThreads, L::kSharedBytes, stream, splits, key_map,
                         value_map, params);
}

template <uint32_t KC>
cudaError_t launch_keys(cudaStream_t stream, const StackAttentionLaunch& launch, uint32_t splits) {
    switch ((launch.shape.vdim + 63) / 64) {
        case 1: return launch_sized<KC, 1>(stream, launch, splits);
        case 2: return launch_sized<KC, 2>(stream, launch, splits);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

// CTAs per token and head over the key axis: enough to fill the machine twice while every warp keeps two pages.
uint32_t stack_attention_splits(const StackAttentionShape& shape, size_t tokens, size_t context) {
    const size_t visible = shape.chunk != 0 ? std::min<size_t>(context, shape.chunk) : context;
    const size_t pages = (visible + kPageSize - 1) / kPageSize;
    uint32_t splits = 1;
    while (splits < 8 && tokens * shape.kv_heads * splits * 2 <= 2 * 148 && pages >= 2 * kWarps * splits * 2) splits *= 2;
    return splits;
}

bool stack_attention_decode_supports(const StackAttentionLaunch& launch) {
    const StackAttentionShape& shape = launch.shape;
    return paged_copies_possible(launch) && shape.dim <= 256 && shape.vdim <= 128 &&
           shape.heads / shape.kv_heads <= kGroupRows;
}

cudaError_t launch_stack_attention_decode(cudaStream_t stream, const StackAttentionLaunch& launch) {
    const uint32_t splits = stack_attention_splits(launch.shape, launch.decode_tokens, launch.decode_context);
    switch ((launch.shape.dim + 63) / 64) {
        case 1: return launch_keys<1>(stream, launch, splits);
        case 2: return launch_keys<2>(stream, launch, splits);
        case 3: return launch_keys<3>(stream, launch, splits);
        case 4: return launch_keys<4>(stream, launch, splits);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace lfm25
