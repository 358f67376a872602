// Captured steps: a table of CUDA graphs keyed on everything a captured step bakes in, shared by the executors.
//
// A serving loop walks through many batch sizes, so the table is large and its least recently used entry is recycled.
// The first step of a key runs eagerly (library plans, function attributes and symbol lookups happen outside any
// capture), the second is captured, later ones only launch the graph.
#pragma once

#include <cuda_runtime.h>
#include <stdint.h>
#include <string.h>

#include <vector>

#include "../../include/lfm25_b200.h"
#include "kernels.h"

namespace lfm25 {

struct Fnv1a {
    uint64_t state = 1469598103934665603ull;
    void word(uint64_t value) { state = (state ^ value) * 1099511628211ull; }
    template <typename Value>
    void add(const Value& value) {   // values of up to 8 bytes are mixed in one step, longer ones word by word
        static_assert(sizeof(Value) % 4 == 0, "hashed fields are 4-byte multiples");
        const unsigned char* cursor = reinterpret_cast<const unsigned char*>(&value);
        for (size_t offset = 0; offset < sizeof(Value); offset += 4) {
            uint32_t part;
            memcpy(&part, cursor + offset, 4);
            word(part);
        }
    }
};

struct StepKey {
    size_t num_tokens = 0;
    size_t splits = 0;        // host-side choices that change the launches of a step
    uint32_t flags = 0;
    uint64_t signature = 0;   // of everything else the graph bakes in
    bool operator==(const StepKey& other) const {
        return num_tokens == other.num_tokens && splits == other.splits && flags == other.flags &&
               signature == other.signature;
    }
};

class StepGraphs {
  public:
    ~StepGraphs() {
        for (Entry& entry : entries_) {
            if (entry.exec != nullptr) cudaGraphExecDestroy(entry.exec);
        }
    }

    // Runs the step of `key`: `enqueue` (returning an LFM25 code) eagerly or under capture, or the captured graph.
    template <typename Enqueue>
    int32_t run(const StepKey& key, cudaStream_t stream, Enqueue enqueue) {
        if (stream == nullptr || stream == cudaStreamLegacy) {
            return report_error(LFM25_ERR_INVALID_ARGUMENT,
                                "graph replay needs the BlasLt handle bound to a non-default stream");
        }
        Entry& entry = find(key);
        entry.last_used = ++clock_;
        if (!entry.warmed) {
            entry.warmed = true;
            return enqueue();
        }
        if (entry.exec == nullptr) {
            const int32_t rc = capture(entry, stream, enqueue);
            if (rc != LFM25_OK) return rc;
        }
        const cudaError_t status = cudaGraphLaunch(entry.exec, stream);
        if (status != cudaSuccess) return failure(status);
        last_kernel_nodes_ = entry.kernel_nodes;
        return LFM25_OK;
    }

    size_t captures() const { return captures_; }
    size_t last_kernel_nodes() const { return last_kernel_nodes_; }   // of the graph launched most recently

  private:
    struct Entry {
        StepKey key;
        bool used = false;
        bool warmed = false;
        cudaGraphExec_t exec = nullptr;
        size_t kernel_nodes = 0;
        uint64_t last_used = 0;
    };

    static int32_t failure(cudaError_t status) { return report_error(LFM25_ERR_CUDA, cudaGetErrorString(status)); }

    Entry& find(const StepKey& key) {
        Entry* victim = nullptr;
        for (Entry& entry : entries_) {
            if (entry.used && entry.key == key) return entry;
            if (victim == nullptr || (victim->used && (!entry.used || entry.last_used < victim->last_used))) {
                victim = &entry;
            }
        }
        if (victim->exec != nullptr) cudaGraphExecDestroy(victim->exec);
        *victim = Entry();
        victim->key = key;
        victim->used = true;
        return *victim;
    }

    template <typename Enqueue>
    int32_t capture(Entry& entry, cudaStream_t stream, Enqueue enqueue) {
        cudaError_t status = cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal);
        if (status != cudaSuccess) return failure(status);
        const int32_t rc = enqueue();
        cudaGraph_t graph = nullptr;
        status = cudaStreamEndCapture(stream, &graph);
        if (rc != LFM25_OK) {
            if (graph != nullptr) cudaGraphDestroy(graph);
            return rc;
        }
        if (status != cudaSuccess) return failure(status);
        size_t node_count = 0;
        if (cudaGraphGetNodes(graph, nullptr, &node_count) == cudaSuccess && node_count > 0) {
            std::vector<cudaGraphNode_t> nodes(node_count);
            if (cudaGraphGetNodes(graph, nodes.data(), &node_count) == cudaSuccess) {
                for (size_t node = 0; node < node_count; ++node) {
                    cudaGraphNodeType type;
                    if (cudaGraphNodeGetType(nodes[node], &type) == cudaSuccess && type == cudaGraphNodeTypeKernel) {
                        ++entry.kernel_nodes;
                    }
                }
            }
        }
        status = cudaGraphInstantiate(&entry.exec, graph, 0);
        cudaGraphDestroy(graph);
        if (status != cudaSuccess) {
            entry.exec = nullptr;
            return failure(status);
        }
        ++captures_;
        return LFM25_OK;
    }

    Entry entries_[96];
    uint64_t clock_ = 0;
    size_t last_kernel_nodes_ = 0;
    size_t captures_ = 0;
};

}  // namespace lfm25
