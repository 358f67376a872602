// Prompt attention of the layer stack on the 5th-generation tensor cores (tcgen05 + tensor memory), for bf16 activations,
// any grouping of query heads, query/key sizes up to 256, value sizes up to 128 and an optional chunk mask.
//
// One CTA owns up to 128 rows of one key/value head: TOKENS consecutive tokens of a segment times the group of query
// heads that share the head.  The roles are those of the LFM2 mixed-step kernel:
//   warp 0      producer: the query tile (one 3-D TMA copy per 64 dimensions: 64 x group x tokens), then the visible key
//               range in stages of 64 keys (4 pages), K chunk by chunk, then V; sizes that are no multiple of 64 are
//               filled up with zeros by the copy
//   warp 1      tensor memory and the MMAs: S = Q K^T (f32), then PV = P V with P read from tensor memory
//   warps 2-5   one thread per row: mask, online softmax with f32 weights, and the running output
// The softmax weights enter the tensor core as a sum of two bf16 values, w = hi + lo, so that they keep 16 significant
// bits; the denominator sums the unrounded weights.
//
// Latent attention takes the same kernel for its prompts (EXPANDED): keys and values of every head have been formed in
// contiguous rows from the latents of the whole context, so a stage is one copy per 64 dimensions instead of one per page,
// the leading key chunks hold a head's own part and the trailing ones the rotated part that all heads share, and the
// output is gated on its way out.
#include <cuda.h>

#include "common.cuh"
#include "launch.h"
#include "stack_attention.h"
#include "stack_common.cuh"
#include "stack_latent.h"
#include "tcgen05.cuh"
#include "tensor_map.h"

namespace lfm25 {

namespace {

constexpr uint32_t kRows = 128;                              // UMMA M
constexpr uint32_t kThreads = 192;
constexpr uint32_t kPagesPerStage = 4;                       // 64 keys
constexpr uint32_t kKeys = kPagesPerStage * kPageSize;
constexpr uint32_t kBoxBytes = kPageSize * 128;              // one page, 64 dimensions: 2 KiB
constexpr uint32_t kChunkBytes = kPagesPerStage * kBoxBytes; // a stage's keys, 64 dimensions: 8 KiB
constexpr uint32_t kQueryChunkBytes = kRows * 128;           // 16 KiB
constexpr uint32_t kControlBytes = 256;

template <uint32_t KC, uint32_t VC>
struct Layout {
    static constexpr uint32_t kStageBytes = (KC + VC) * kChunkBytes;
    static constexpr uint32_t kStages = KC + VC <= 2 ? 4 : 3;
    static constexpr uint32_t kSharedBytes = KC * kQueryChunkBytes + kStages * kStageBytes + kControlBytes + 1024;
    static constexpr uint32_t kColumnPv = 2 * kKeys;         // two S buffers in front, two PV buffers behind
    static constexpr uint32_t kTmemColumns = 2 * kKeys + 2 * 64 * VC <= 256 ? 256 : 512;
    static constexpr uint32_t kCtasPerSm = VC == 1 && kTmemColumns <= 256 && kSharedBytes <= 112 * 1024 ? 2 : 1;
    static_assert(2 * kKeys + 2 * 64 * VC <= 512, "tensor memory");
    static_assert(kSharedBytes <= 227 * 1024, "shared memory");
};

struct Params {
    StackAttentionShape shape;
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* positions;
    StackSegments segments;
    __nv_bfloat16* out;
    size_t out_pitch;
    unsigned int* status;
    uint32_t tile_tokens;
    // EXPANDED: shape.kv_heads == shape.heads
    uint32_t own_chunks;           // 64-dimension key chunks of a head's own part; the others are the shared part
    uint32_t own_dim;              // first query dimension of the shared part
    const uint32_t* bases;         // first row of each segment's context
    const __nv_bfloat16* gate;     // token t, head h at gate + t * gate_pitch + h * vdim
    size_t gate_pitch;
};

__device__ __forceinline__ void mma_smem(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc,
                                         uint32_t accumulate) {
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
        "}\n" ::"r"(tmem_d),
        "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void mma_tmem(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc,
                                         uint32_t accumulate) {
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n"
        "}\n" ::"r"(tmem_d),
        "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void tma_load_box_3d(uint32_t dst, const void* tensor_map, uint32_t bar, int32_t x, int32_t y,
                                                int32_t z) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
        ::"r"(dst), "l"(reinterpret_cast<uint64_t>(tensor_map)), "r"(bar), "r"(x), "r"(y), "r"(z)
        : "memory");
}

// A weight pair as two bf16 pairs whose sum carries 16 bits of each weight.
__device__ __forceinline__ void split_weights(float a, float b, uint32_t& high, uint32_t& low) {
    high = pack_bf16x2(a, b);
    const float2 rounded = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high));
    low = pack_bf16x2(a - rounded.x, b - rounded.y);
}

template <uint32_t KC, uint32_t VC, bool EXPANDED>
__global__ void __launch_bounds__(kThreads, Layout<KC, VC>::kCtasPerSm)
stack_attention_umma_kernel(const __grid_constant__ CUtensorMap query_map, const __grid_constant__ CUtensorMap key_map,
                            const __grid_constant__ CUtensorMap value_map, const __grid_constant__ CUtensorMap shared_map,
                            const Params p) {
    using L = Layout<KC, VC>;
    const uint32_t warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0);     // the same value to the compiler's eye as well
    const uint32_t lane = threadIdx.x & 31;
    pdl_launch_dependents();
    pdl_wait();

    // later tiles tend to have longer key ranges, so the grid runs backwards
    const uint32_t kv_head = blockIdx.x % p.shape.kv_heads;
    const SegmentTile tile =
        locate_tile(p.segments, p.tile_tokens, (gridDim.x - 1 - blockIdx.x) / p.shape.kv_heads);
    if (tile.count == 0) {
        return;
    }
    const uint32_t group = p.shape.heads / p.shape.kv_heads;
    const uint32_t first_position = p.positions[tile.first];
    const uint32_t last_position = first_position + tile.count - 1;
    const uint32_t* __restrict__ table = nullptr;
    uint32_t first_page = 0;
    uint32_t context_row = 0;
    uint32_t pages = last_position / kPageSize + 1;
    if constexpr (EXPANDED) {
        context_row = p.bases[tile.segment];
        pages = (pages + kPagesPerStage - 1) / kPagesPerStage * kPagesPerStage;     // contexts end on whole stages
    } else {
        const size_t table_row = p.segments.slots[tile.segment];
        if (table_row >= p.block_table_rows || last_position / kPageSize >= p.block_table_stride) {
            return;
        }
        table = p.block_tables + table_row * p.block_table_stride;
        first_page = first_visible(first_position, p.shape.chunk) / kPageSize;
        pages -= first_page;
    }
    const uint32_t stages_total = (pages + kPagesPerStage - 1) / kPagesPerStage;

    extern __shared__ uint8_t attention_smem[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(attention_smem) + 1023) & ~uintptr_t(1023));
    const uint32_t q_base = smem_u32(smem);
    const uint32_t ring = q_base + KC * kQueryChunkBytes;
    uint8_t* control = smem + KC * kQueryChunkBytes + L::kStages * L::kStageBytes;
    const uint32_t bar_full = smem_u32(control);
    const uint32_t bar_empty = bar_full + 8 * L::kStages;
    const uint32_t bar_q = bar_empty + 8 * L::kStages;
    const uint32_t bar_s = bar_q + 8;      // [2]: S of an even / odd stage is complete
    const uint32_t bar_p = bar_s + 16;     // [2]: its weights are in tensor memory
    const uint32_t bar_pv = bar_p + 16;    // [2]: its PV product is complete
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(control + 8 * (2 * L::kStages + 7));
    volatile uint32_t* flags = tmem_slot + 1;   // [0] unassigned page met, [1] abort

    if (threadIdx.x == 0) {
        tma_prefetch_descriptor(&query_map);
        tma_prefetch_descriptor(&key_map);
        tma_prefetch_descriptor(&value_map);
        if constexpr (EXPANDED) tma_prefetch_descriptor(&shared_map);
        for (uint32_t stage = 0; stage < L::kStages; ++stage) {
            mbar_init(bar_full + 8 * stage, 1);
            mbar_init(bar_empty + 8 * stage, 1);
        }
        mbar_init(bar_q, 1);
        for (uint32_t buffer = 0; buffer < 2; ++buffer) {
            mbar_init(bar_s + 8 * buffer, 1);
            mbar_init(bar_p + 8 * buffer, 4);
            mbar_init(bar_pv + 8 * buffer, 1);
        }
        flags[0] = 0;
        flags[1] = 0;
        fence_barrier_init();
        fence_proxy_async_smem();
    }
    if (warp == 1) {
        tmem_allocate(smem_u32(const_cast<uint32_t*>(tmem_slot)), L::kTmemColumns);
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        // ------------------------------------------------------------------------------------ producer
        if (elect_one()) {
            mbar_arrive_expect_tx(bar_q, KC * group * p.tile_tokens * 128);
            for (uint32_t chunk = 0; chunk < KC; ++chunk) {
                // a query dimension beyond a part of the head meets a key dimension that the copy filled with zero
                const bool shared_part = EXPANDED && chunk >= p.own_chunks;
                const uint32_t x = shared_part ? p.own_dim + (chunk - p.own_chunks) * 64 : chunk * 64;
                tma_load_box_3d(q_base + chunk * kQueryChunkBytes, &query_map, bar_q, static_cast<int32_t>(x),
                                static_cast<int32_t>(kv_head * group), static_cast<int32_t>(tile.first));
            }
            for (uint32_t index = 0; index < stages_total; ++index) {
                const uint32_t stage = index % L::kStages;
                if (index >= L::kStages) {
                    if (flags[1] || !mbar_wait_bounded(bar_empty + 8 * stage, ((index / L::kStages) - 1) & 1)) {
                        if (!flags[1]) {
                            flags[1] = 1;
                            record_wait_timeout(p.status, kTagStackAttention, (blockIdx.x << 2) | 1);
                        }
                        break;
                    }
                }
                const uint32_t bar = bar_full + 8 * stage;
                const uint32_t count = min(kPagesPerStage, pages - index * kPagesPerStage);
                if constexpr (EXPANDED) {
                    const int32_t row = static_cast<int32_t>(context_row + index * kKeys);
                    const int32_t head = static_cast<int32_t>(kv_head);
                    const uint32_t target = ring + stage * L::kStageBytes;
                    mbar_arrive_expect_tx(bar, L::kStageBytes);
#pragma unroll
                    for (uint32_t chunk = 0; chunk < KC; ++chunk) {
                        if (chunk < p.own_chunks) {
                            tma_load_box_3d(target + chunk * kChunkBytes, &key_map, bar, static_cast<int32_t>(chunk * 64),
                                            head, row);
                        } else {
                            tma_load_2d(target + chunk * kChunkBytes, &shared_map, bar,
                                        static_cast<int32_t>((chunk - p.own_chunks) * 64), row);
                        }
                    }
#pragma unroll
                    for (uint32_t chunk = 0; chunk < VC; ++chunk) {
                        tma_load_box_3d(target + (KC + chunk) * kChunkBytes, &value_map, bar,
                                        static_cast<int32_t>(chunk * 64), head, row);
                    }
                    continue;
                }
                // an unassigned page is flagged before anything of the stage is announced, and page 0 is read in its
                // place so that the pipeline stays uniform
                uint32_t entries[kPagesPerStage];
#pragma unroll
                for (uint32_t sub = 0; sub < kPagesPerStage; ++sub) {
                    entries[sub] = 0;
                    if (sub < count) {
                        entries[sub] = __ldg(table + first_page + index * kPagesPerStage + sub);
                        if (entries[sub] >= p.num_pages) {
                            flags[0] = 1;
                            entries[sub] = 0;
                        }
                    }
                }
                mbar_arrive_expect_tx(bar, count * (KC + VC) * kBoxBytes);
#pragma unroll
                for (uint32_t sub = 0; sub < kPagesPerStage; ++sub) {
                    if (sub >= count) {
                        continue;
                    }
                    const int32_t row = static_cast<int32_t>((entries[sub] * p.shape.kv_heads + kv_head) * kPageSize);
                    const uint32_t target = ring + stage * L::kStageBytes + sub * kBoxBytes;
#pragma unroll
                    for (uint32_t chunk = 0; chunk < KC; ++chunk) {
                        tma_load_2d(target + chunk * kChunkBytes, &key_map, bar, static_cast<int32_t>(chunk * 64), row);
                    }
#pragma unroll
                    for (uint32_t chunk = 0; chunk < VC; ++chunk) {
                        tma_load_2d(target + (KC + chunk) * kChunkBytes, &value_map, bar,
                                    static_cast<int32_t>(chunk * 64), row);
                    }
                }
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------------------------------ MMA issuer
        if (elect_one()) {
            // D = f32, A = B = bf16, M = 128; S: both K-major, N = keys of the stage; PV: B (the V rows) MN-major, N = 64
            const uint32_t idesc_common = (1u << 4) | (1u << 7) | (1u << 10) | ((kRows >> 4) << 24);
            const uint32_t idesc_pv = idesc_common | (1u << 16) | ((64u >> 3) << 17);
            bool ok = !flags[1] && mbar_wait_bounded(bar_q, 0);
            if (!ok && !flags[1]) {
                flags[1] = 1;
                record_wait_timeout(p.status, kTagStackAttention, (blockIdx.x << 2) | 2);
            }
            auto issue_scores = [&](uint32_t index) -> bool {
                const uint32_t stage = index % L::kStages;
                const uint32_t count = min(kPagesPerStage, pages - index * kPagesPerStage);
                if (flags[1] || !mbar_wait_bounded(bar_full + 8 * stage, (index / L::kStages) & 1)) {
                    return false;
                }
                tcgen05_fence_after();
                const uint32_t idesc_qk = idesc_common | (((count * kPageSize) >> 3) << 17);
                const uint32_t target = tmem_base + (index & 1) * kKeys;
#pragma unroll
                for (uint32_t chunk = 0; chunk < KC; ++chunk) {
                    const uint64_t q_desc = smem_descriptor(q_base + chunk * kQueryChunkBytes);
                    const uint64_t k_desc = smem_descriptor(ring + stage * L::kStageBytes + chunk * kChunkBytes);
#pragma unroll
                    for (uint32_t ks = 0; ks < 4; ++ks) {   // 16 dimensions = 32 bytes inside the swizzled row per step
                        mma_smem(target, q_desc + ks * 2, k_desc + ks * 2, idesc_qk, chunk + ks);
                    }
                }
                umma_commit(bar_s + 8 * (index & 1));
                return true;
            };
            ok = ok && issue_scores(0);
            for (uint32_t index = 0; index < stages_total && ok; ++index) {
                const uint32_t stage = index % L::kStages;
                const uint32_t count = min(kPagesPerStage, pages - index * kPagesPerStage);
                const uint32_t buffer = index & 1;
                // the next stage's scores first: the tensor core computes them while this stage's softmax runs.  Their
                // buffer is free: its previous weights were consumed by the PV product issued before, and MMAs execute
                // in issue order.
                if (index + 1 < stages_total && !issue_scores(index + 1)) {
                    ok = false;
                    break;
                }
                if (flags[1] || !mbar_wait_bounded(bar_p + 8 * buffer, (index >> 1) & 1)) {
                    ok = false;
                    break;
                }
                tcgen05_fence_after();
                for (uint32_t step = 0; step < count; ++step) {   // 16 keys: 8 packed columns of P, 2 KiB of V
                    const uint32_t weights = tmem_base + buffer * kKeys + step * 8;
#pragma unroll
                    for (uint32_t chunk = 0; chunk < VC; ++chunk) {
                        const uint64_t v_desc = smem_descriptor(ring + stage * L::kStageBytes +
                                                                (KC + chunk) * kChunkBytes + step * kBoxBytes);
                        const uint32_t target = tmem_base + L::kColumnPv + (buffer * VC + chunk) * 64;
                        mma_tmem(target, weights, v_desc, idesc_pv, step);
                        mma_tmem(target, weights + kKeys / 2, v_desc, idesc_pv, 1);
                    }
                }
                umma_commit(bar_pv + 8 * buffer);
                umma_commit(bar_empty + 8 * stage);
            }
            if (!ok && !flags[1]) {
                flags[1] = 1;
                record_wait_timeout(p.status, kTagStackAttention, (blockIdx.x << 2) | 3);
            }
        }
    } else {
        // ------------------------------------------------------------------------------------ softmax / output
        const uint32_t quadrant = warp & 3;                 // the tensor-memory lanes this warp may touch
        const uint32_t row = quadrant * 32 + lane;
        const uint32_t token = row / group;                 // of the tile
        const uint32_t head = row - token * group;
        const bool live = token < tile.count;
        // rows without a token follow the last one, so that they never hold back the mask-free path
        const int32_t row_position = static_cast<int32_t>(live ? first_position + token : last_position);
        const int32_t row_first = static_cast<int32_t>(first_visible(row_position, p.shape.chunk));
        const uint32_t lane_address = tmem_base + ((quadrant * 32) << 16);
        const uint32_t softmax_thread = threadIdx.x - 64;   // 0..127, for cooperative shared-memory writes
        const float scale_log2 = p.shape.scale * kLog2e;
        float running_max = -INFINITY;
        float running_sum = 0.0f;
        float out[64 * VC];
#pragma unroll
        for (uint32_t dim = 0; dim < 64 * VC; ++dim) out[dim] = 0.0f;
        bool ok = true;
        // O <- (O + PV of stage `index`) * factor: the PV product is folded in one stage late
        auto fold = [&](uint32_t index, float factor) -> bool {
            const bool ready = !flags[1] && mbar_wait_bounded(bar_pv + 8 * (index & 1), (index >> 1) & 1);
            if (!__all_sync(0xffffffffu, ready)) {
                return false;
            }
            tcgen05_fence_after();
            const uint32_t source = lane_address + L::kColumnPv + (index & 1) * VC * 64;
            const bool unchanged = __all_sync(0xffffffffu, factor == 1.0f);
#pragma unroll
            for (uint32_t half = 0; half < 2 * VC; ++half) {
                uint32_t raw[2][16];
                tmem_load16_nowait(source + half * 32, raw[0]);
                tmem_load16_nowait(source + half * 32 + 16, raw[1]);
                tmem_load_wait();
                if (unchanged) {
#pragma unroll
                    for (uint32_t j = 0; j < 32; ++j) out[half * 32 + j] += __uint_as_float(raw[j >> 4][j & 15]);
                } else {
#pragma unroll
                    for (uint32_t j = 0; j < 32; ++j) {
                        out[half * 32 + j] = (out[half * 32 + j] + __uint_as_float(raw[j >> 4][j & 15])) * factor;
                    }
                }
            }
            return true;
        };
        for (uint32_t index = 0; index < stages_total; ++index) {
            const uint32_t stage = index % L::kStages;
            const uint32_t buffer = index & 1;
            ok = !flags[1] && mbar_wait_bounded(bar_s + 8 * buffer, (index >> 1) & 1);
            if (!__all_sync(0xffffffffu, ok)) {
                ok = false;
                break;
            }
            tcgen05_fence_after();
            const uint32_t scores = lane_address + buffer * kKeys;
            const int32_t stage_first = static_cast<int32_t>((first_page + index * kPagesPerStage) * kPageSize);
            // keys of this stage that the row sees: from .. to - 1
            const int32_t from = row_first - stage_first;
            const int32_t to = row_position - stage_first + 1;
            const bool fast = __all_sync(0xffffffffu, from <= 0 && to >= static_cast<int32_t>(kKeys));
            float lane_max[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                uint32_t raw[2][16];
                tmem_load16_nowait(scores + half * 32, raw[0]);
                tmem_load16_nowait(scores + half * 32 + 16, raw[1]);
                tmem_load_wait();
                if (fast) {
#pragma unroll
                    for (uint32_t j = 0; j < 32; ++j) {
                        lane_max[j & 3] = fmaxf(lane_max[j & 3], __uint_as_float(raw[j >> 4][j & 15]));
                    }
                } else {
#pragma unroll
                    for (uint32_t j = 0; j < 32; ++j) {
                        const int32_t key = static_cast<int32_t>(half * 32 + j);
                        if (key >= from && key < to) {
                            lane_max[j & 3] = fmaxf(lane_max[j & 3], __uint_as_float(raw[j >> 4][j & 15]));
                        }
                    }
                }
            }
            const float new_max =
                fmaxf(running_max, fmaxf(fmaxf(lane_max[0], lane_max[1]), fmaxf(lane_max[2], lane_max[3])));
            const float base = new_max == -INFINITY ? 0.0f : new_max;     // nothing visible so far: all weights are zero
            const float rescale = fast_exp2((running_max - base) * scale_log2);
            const float offset = -base * scale_log2;
            float lane_sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            uint32_t low[2][16];     // the low parts of the first half may only be written once the second half is read
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                uint32_t raw[2][16];
                tmem_load16_nowait(scores + half * 32, raw[0]);
                tmem_load16_nowait(scores + half * 32 + 16, raw[1]);
                tmem_load_wait();
                uint32_t high[16];
#pragma unroll
                for (uint32_t j = 0; j < 32; j += 2) {
                    const int32_t key = static_cast<int32_t>(half * 32 + j);
                    float w0 = fast_exp2(fmaf(__uint_as_float(raw[j >> 4][j & 15]), scale_log2, offset));
                    float w1 = fast_exp2(fmaf(__uint_as_float(raw[j >> 4][(j & 15) + 1]), scale_log2, offset));
                    if (!fast) {
                        w0 = key >= from && key < to ? w0 : 0.0f;
                        w1 = key + 1 >= from && key + 1 < to ? w1 : 0.0f;
                    }
                    split_weights(w0, w1, high[j / 2], low[half][j / 2]);
                    lane_sum[(j >> 1) & 3] += w0 + w1;
                }
                tmem_store16(scores + half * 16, high);
            }
            tmem_store16(scores + kKeys / 2, low[0]);
            tmem_store16(scores + kKeys / 2 + 16, low[1]);
            const float stage_sum = (lane_sum[0] + lane_sum[1]) + (lane_sum[2] + lane_sum[3]);
            tmem_store_wait();
            // V rows of keys that no token of the tile has may hold anything: clear them (a zero weight times a NaN
            // pattern is NaN)
            const int32_t exists = static_cast<int32_t>(last_position) - stage_first + 1;
            if (exists < static_cast<int32_t>(kKeys)) {
                const uint32_t v_base = ring + stage * L::kStageBytes + KC * kChunkBytes;
                const uint32_t count = min(kPagesPerStage, pages - index * kPagesPerStage);
                for (uint32_t item = softmax_thread; item < kKeys * 8 * VC; item += 128) {
                    const uint32_t chunk = item / (kKeys * 8);
                    const uint32_t key = item / 8 % kKeys;
                    if (static_cast<int32_t>(key) >= exists && key < count * kPageSize) {
                        asm volatile("st.shared.v4.u32 [%0], {%1, %1, %1, %1};" ::"r"(v_base + chunk * kChunkBytes +
                                                                                      key * 128 + item % 8 * 16),
                                     "r"(0u)
                                     : "memory");
                    }
                }
                fence_proxy_async_smem();
            }
            tcgen05_fence_before();
            __syncwarp();
            if (lane == 0) {
                mbar_arrive(bar_p + 8 * buffer);
            }
            // fold in the previous stage's PV product (computed with the previous maximum): it and the accumulator move
            // to the new maximum together
            if (index > 0 && !fold(index - 1, rescale)) {
                ok = false;
                break;
            }
            running_sum = fmaf(running_sum, rescale, stage_sum);
            running_max = new_max;
        }
        if (ok) {
            ok = fold(stages_total - 1, 1.0f);
        }
        if (!ok && lane == 0 && !flags[1]) {
            flags[1] = 1;
            record_wait_timeout(p.status, kTagStackAttention, (blockIdx.x << 2) | 0);
        }
        if (ok && live && flags[0] == 0 && flags[1] == 0) {
            const float inverse = 1.0f / running_sum;
            __nv_bfloat16* target = p.out + static_cast<size_t>(tile.first + token) * p.out_pitch +
                                    (static_cast<size_t>(kv_head) * group + head) * p.shape.vdim;
#pragma unroll
            for (uint32_t part = 0; part < 8 * VC; ++part) {
                if (part * 8 < p.shape.vdim) {      // vdim is a multiple of 8
                    if constexpr (EXPANDED) {
                        float gate[8];
                        load_values<8>(p.gate + static_cast<size_t>(tile.first + token) * p.gate_pitch +
                                           kv_head * p.shape.vdim + part * 8,
                                       gate);
#pragma unroll
                        for (uint32_t i = 0; i < 8; ++i) out[part * 8 + i] *= 1.0f / (1.0f + __expf(-gate[i]));
                    }
                    uint4 value;
                    value.x = pack_bf16x2(out[part * 8] * inverse, out[part * 8 + 1] * inverse);
                    value.y = pack_bf16x2(out[part * 8 + 2] * inverse, out[part * 8 + 3] * inverse);
                    value.z = pack_bf16x2(out[part * 8 + 4] * inverse, out[part * 8 + 5] * inverse);
                    value.w = pack_bf16x2(out[part * 8 + 6] * inverse, out[part * 8 + 7] * inverse);
                    *reinterpret_cast<uint4*>(target + part * 8) = value;
                }
            }
        }
    }

    // the producer and MMA warps ran their loops on one lane: the warp meets again here, so that the CTA barrier below
    // is reached by whole warps
    __syncwarp();
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tmem_free(tmem_base, L::kTmemColumns);
    }
}

// (dimensions, heads, tokens) with boxes of 64 x group x tokens
bool make_query_map(CUtensorMap* map, const StackAttentionLaunch& launch, uint32_t group, uint32_t tile_tokens) {
    EncodeTiledFn encode = encode_tiled_entry();
    if (encode == nullptr) {
        return false;
    }
    const cuuint64_t dim = launch.shape.dim, heads = launch.shape.heads;
    const cuuint64_t dims[3] = {dim, heads, launch.segments.num_tokens};
    const cuuint64_t strides[2] = {dim * 2, heads * dim * 2};
    const cuuint32_t box[3] = {64, group, tile_tokens};
    const cuuint32_t element_strides[3] = {1, 1, 1};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(launch.query), dims, strides, box,
                  element_strides, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                  CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <uint32_t KC, uint32_t VC, bool EXPANDED>
cudaError_t launch_maps(cudaStream_t stream, const CUtensorMap& query_map, const CUtensorMap& key_map,
                        const CUtensorMap& value_map, const CUtensorMap& shared_map, const Params& params) {
    using L = Layout<KC, VC>;
    const auto kernel = stack_attention_umma_kernel<KC, VC, EXPANDED>;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                    static_cast<int>(L::kSharedBytes));
    if (status != cudaSuccess) return status;
    const size_t tiles = tile_bound(params.segments, params.tile_tokens);
    return launch_kernel(kernel, static_cast<unsigned int>(tiles * params.shape.kv_heads), kThreads, L::kSharedBytes,
                         stream, 1, query_map, key_map, value_map, shared_map, params);
}

// `key_chunks` and `value_chunks` of 64 dimensions
template <bool EXPANDED>
cudaError_t launch_chunks(cudaStream_t stream, uint32_t key_chunks, uint32_t value_chunks, const CUtensorMap& query_map,
                          const CUtensorMap& key_map, const CUtensorMap& value_map, const CUtensorMap& shared_map,
                          const Params& params) {
    auto go = [&](auto narrow, auto wide) {
        return (value_chunks > 1 ? wide : narrow)(stream, query_map, key_map, value_map, shared_map, params);
    };
    switch (key_chunks) {
        case 1: return go(launch_maps<1, 1, EXPANDED>, launch_maps<1, 2, EXPANDED>);
        case 2: return go(launch_maps<2, 1, EXPANDED>, launch_maps<2, 2, EXPANDED>);
        case 3: return go(launch_maps<3, 1, EXPANDED>, launch_maps<3, 2, EXPANDED>);
        case 4: return go(launch_maps<4, 1, EXPANDED>, launch_maps<4, 2, EXPANDED>);
        default: return cudaErrorInvalidValue;
    }
}

// [rows, heads, size] with the heads of a row side by side and rows `pitch` elements apart, in boxes of 64 dimensions of
// one head x `box_rows`
bool make_head_map(CUtensorMap* map, const void* base, size_t size, size_t heads, size_t rows, size_t pitch,
                   uint32_t box_rows) {
    EncodeTiledFn encode = encode_tiled_entry();
    if (encode == nullptr) {
        return false;
    }
    const cuuint64_t dims[3] = {size, heads, rows};
    const cuuint64_t strides[2] = {size * 2, pitch * 2};
    const cuuint32_t box[3] = {64, 1, box_rows};
    const cuuint32_t element_strides[3] = {1, 1, 1};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, element_strides,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

uint32_t chunks_of(uint32_t size) { return (size + 63) / 64; }

}  // namespace

bool make_page_map(CUtensorMap* map, const StackAttentionLaunch& launch, bool value) {
    const uint64_t rows = static_cast<uint64_t>(launch.num_pages) * launch.shape.kv_heads * kPageSize;
    const uint64_t size = value ? launch.shape.vdim : launch.shape.dim;
    return make_swizzled_2d_map_width(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2,
                                      value ? launch.value_cache : launch.key_cache, rows, size, size * 2, kPageSize);
}

bool paged_copies_possible(const StackAttentionLaunch& launch) {
    const StackAttentionShape& shape = launch.shape;
    return launch.type == Activation::kBf16 && launch.status != nullptr && shape.dim % 8 == 0 && shape.vdim % 8 == 0 &&
           shape.scale > 0.0f && launch.out_pitch % 8 == 0 && aligned_to(launch.query, 16) &&
           aligned_to(launch.key_cache, 16) && aligned_to(launch.value_cache, 16) && aligned_to(launch.out, 16) &&
           static_cast<uint64_t>(launch.num_pages) * shape.kv_heads * kPageSize <= 0x7fffffffu;
}

bool stack_attention_umma_supports(const StackAttentionLaunch& launch) {
    const StackAttentionShape& shape = launch.shape;
    return paged_copies_possible(launch) && shape.dim <= 256 && shape.vdim <= 128 &&
           shape.heads / shape.kv_heads <= kRows && launch.segments.offsets != nullptr;
}

cudaError_t launch_stack_attention_umma(cudaStream_t stream, const StackAttentionLaunch& launch) {
    const StackAttentionShape& shape = launch.shape;
    const uint32_t group = shape.heads / shape.kv_heads;
    Params params = {};
    params.shape = shape;
    params.block_tables = launch.block_tables;
    params.block_table_stride = launch.block_table_stride;
    params.block_table_rows = launch.block_table_rows;
    params.num_pages = launch.num_pages;
    params.positions = launch.positions;
    params.segments = launch.segments;
    params.out = static_cast<__nv_bfloat16*>(launch.out);
    params.out_pitch = launch.out_pitch;
    params.status = launch.status;
    params.tile_tokens = kRows / group;
    CUtensorMap query_map, key_map, value_map;
    if (!make_query_map(&query_map, launch, group, params.tile_tokens) || !make_page_map(&key_map, launch, false) ||
        !make_page_map(&value_map, launch, true)) {
        return cudaErrorInvalidValue;
    }
    return launch_chunks<false>(stream, chunks_of(shape.dim), chunks_of(shape.vdim), query_map, key_map, value_map, key_map,
                                params);
}

bool expanded_attention_supports(Activation type, const LatentAttentionShape& shape, size_t out_pitch, size_t gate_pitch,
                                 size_t expanded_pitch) {
    return type == Activation::kBf16 && shape.scale > 0.0f && shape.dim % 8 == 0 && shape.rot_dim % 8 == 0 &&
           shape.vdim % 8 == 0 && shape.kv_rank % 8 == 0 && shape.vdim <= 128 &&
           chunks_of(shape.dim) + chunks_of(shape.rot_dim) <= 4 && out_pitch % 8 == 0 && gate_pitch % 8 == 0 &&
           expanded_pitch % 8 == 0;
}

cudaError_t launch_expanded_attention(cudaStream_t stream, const ExpandedAttentionLaunch& launch) {
    const LatentAttentionShape& shape = launch.shape;
    Params params = {};
    params.shape = {shape.heads, shape.heads, shape.dim + shape.rot_dim, shape.vdim, 0, 0, shape.scale};
    params.positions = launch.positions;
    // segment offsets are absolute token indices, so leaving segments out is simply a later start
    params.segments = launch.segments;
    params.segments.offsets += launch.first_segment;
    params.segments.slots += launch.first_segment;
    params.segments.num_segments -= launch.first_segment;
    params.out = static_cast<__nv_bfloat16*>(launch.out);
    params.out_pitch = launch.out_pitch;
    params.status = launch.status;
    params.tile_tokens = kRows;
    params.own_chunks = chunks_of(shape.dim);
    params.own_dim = shape.dim;
    params.bases = launch.bases + launch.first_segment;
    params.gate = static_cast<const __nv_bfloat16*>(launch.gate);
    params.gate_pitch = launch.gate_pitch;
    const auto* expanded = static_cast<const __nv_bfloat16*>(launch.expanded);
    CUtensorMap query_map, key_map, value_map, shared_map;
    if (!make_head_map(&query_map, launch.query, shape.dim + shape.rot_dim, shape.heads, launch.segments.num_tokens,
                       launch.query_pitch, kRows) ||
        !make_head_map(&key_map, expanded, shape.dim, shape.heads, launch.rows, launch.expanded_pitch, kKeys) ||
        !make_head_map(&value_map, expanded + static_cast<size_t>(shape.heads) * shape.dim, shape.vdim, shape.heads,
                       launch.rows, launch.expanded_pitch, kKeys) ||
        !make_swizzled_2d_map_width(&shared_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, launch.keys, launch.rows,
                                    shape.rot_dim, shape.rot_dim * 2, kKeys)) {
        return cudaErrorInvalidValue;
    }
    return launch_chunks<true>(stream, params.own_chunks + chunks_of(shape.rot_dim), chunks_of(shape.vdim), query_map,
                               key_map, value_map, shared_map, params);
}

}  // namespace lfm25
