// Pieces shared by the device-resident engines (engine.cu: GPT-2 and Gemma-3, engine_decoder.cu): the owner of an
// engine's device memory and the recorded decode steps.
#pragma once
#include <string.h>

#include <vector>

#include "zq_internal.h"

namespace zq {
namespace {

struct DeviceArena {
    std::vector<void*> ptrs;
    size_t total = 0;
    ~DeviceArena() {
        for (void* p : ptrs) cudaFree(p);
    }
    int alloc(void** out, size_t bytes) {
        cudaError_t e = cudaMalloc(out, bytes ? bytes : 4);
        if (e != cudaSuccess) {
            g_last_cuda_error = (int)e;
            return e == cudaErrorMemoryAllocation ? ZQ_ERR_NO_MEM : ZQ_ERR_CUDA;
        }
        ptrs.push_back(*out);
        total += bytes;
        return ZQ_OK;
    }
    template <typename T>
    int alloc_n(T** out, size_t n) {
        return alloc(reinterpret_cast<void**>(out), n * sizeof(T));
    }
    int upload_f32(float** out, const float* host, size_t n, cudaStream_t st) {
        if (!host) return ZQ_ERR_BAD_ARG;
        int rc = alloc_n(out, n);
        if (rc != ZQ_OK) return rc;
        ZQ_CUDA(cudaMemcpyAsync(*out, host, n * sizeof(float), cudaMemcpyHostToDevice, st));
        return ZQ_OK;
    }
};

// A decode step is a fixed launch sequence whose only varying inputs live in device memory, so it is
// captured once per variant and replayed. The first use of a variant runs eagerly (function
// attributes get set and launch errors surface outside capture); the second captures on the
// engine's own stream (the caller's may be the legacy default stream, which cannot capture); every
// use from then on is one graph launch on the caller's stream.
enum StepVariant { STEP_CACHE_ONLY = 0, STEP_LOGITS = 1, STEP_GREEDY = 2, STEP_BATCH = 3, STEP_VARIANTS = 4 };

struct StepGraphs {
    cudaGraphExec_t exec[STEP_VARIANTS] = {nullptr, nullptr, nullptr, nullptr};
    bool warmed[STEP_VARIANTS] = {false, false, false, false};
    cudaStream_t capture_stream = nullptr;
    bool disabled = false;
    ~StepGraphs() {
        for (cudaGraphExec_t e : exec)
            if (e) cudaGraphExecDestroy(e);
        if (capture_stream) cudaStreamDestroy(capture_stream);
    }
    template <typename Body>
    int run(int variant, cudaStream_t st, Body&& body) {
        if (disabled) return body(st);
        if (!warmed[variant]) {
            warmed[variant] = true;
            return body(st);
        }
        if (!exec[variant]) {
            if (!capture_stream) ZQ_CUDA(cudaStreamCreateWithFlags(&capture_stream, cudaStreamNonBlocking));
            ZQ_CUDA(cudaStreamBeginCapture(capture_stream, cudaStreamCaptureModeThreadLocal));
            const int rc = body(capture_stream);
            cudaGraph_t graph = nullptr;
            const cudaError_t e = cudaStreamEndCapture(capture_stream, &graph);
            if (rc != ZQ_OK || e != cudaSuccess) {
                if (graph) cudaGraphDestroy(graph);
                return rc != ZQ_OK ? rc : cuda_fail(e);
            }
            const cudaError_t ei = cudaGraphInstantiate(&exec[variant], graph, 0);
            cudaGraphDestroy(graph);
            if (ei != cudaSuccess) {
                exec[variant] = nullptr;
                return cuda_fail(ei);
            }
        }
        ZQ_CUDA(cudaGraphLaunch(exec[variant], st));
        return ZQ_OK;
    }
};

}  // namespace
}  // namespace zq
