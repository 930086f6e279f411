// What every library built from this directory needs whatever kernels it carries: the error text, contexts, the
// context's growing device blocks, recorded graphs and plain device memory (include/peregrine_b200.h).
#include <stdarg.h>
#include <string.h>

#include <algorithm>
#include <new>

#include "pg_internal.cuh"

std::atomic<uint64_t> g_pg_launches{0};
static thread_local char g_err[512] = "";

void pg_set_error(const char *fmt, ...)
{
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof(g_err), fmt, ap);
    va_end(ap);
}

// Grows one of the context's device blocks.  Work already enqueued may still use the old block, so the stream is
// drained first; a recorded graph may use it for as long as it lives, so with graphs alive the old block is parked
// (pg_ctx::retired) instead of freed.
static int32_t grow_block(pg_ctx *ctx, void **block, size_t *have, size_t bytes, const char *what, bool zeroed)
{
    if (bytes <= *have) return PG_OK;
    if (ctx->capturing)
        PG_FAIL(PG_ERR_INVALID, "%s memory would have to grow while a graph is being recorded; run the call once before recording", what);
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    if (*block) {
        if (ctx->live_graphs > 0)
            ctx->retired.push_back(*block);
        else
            PG_CUDA(cudaFree(*block));
    }
    *block = nullptr;
    *have = 0;
    size_t want = bytes + (bytes >> 2);
    want = (want + 255) & ~(size_t)255;
    PG_CUDA(cudaMalloc(block, want));
    if (zeroed) PG_CUDA(cudaMemsetAsync(*block, 0, want, ctx->stream));
    *have = want;
    return PG_OK;
}

int32_t pg_scratch_reserve(pg_ctx *ctx, size_t bytes) { return grow_block(ctx, &ctx->scratch, &ctx->scratch_bytes, bytes, "scratch", false); }
int32_t pg_staging_reserve(pg_ctx *ctx, size_t bytes) { return grow_block(ctx, &ctx->staging, &ctx->staging_bytes, bytes, "staging", false); }
int32_t pg_splitk_reserve(pg_ctx *ctx, size_t bytes) { return grow_block(ctx, &ctx->splitk, &ctx->splitk_bytes, bytes, "split-K workspace", true); }

int32_t pg_pinned_reserve(pg_ctx *ctx, size_t bytes)
{
    if (bytes <= ctx->h_pinned_bytes) return PG_OK;
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    if (ctx->h_pinned) PG_CUDA(cudaFreeHost(ctx->h_pinned));
    ctx->h_pinned = nullptr;
    ctx->h_pinned_bytes = 0;
    size_t want = bytes + (bytes >> 2);
    PG_CUDA(cudaMallocHost(&ctx->h_pinned, want));
    ctx->h_pinned_bytes = want;
    return PG_OK;
}

extern "C" {

const char *pg_last_error(void) { return g_err; }
int32_t pg_version(void) { return 100; }
uint64_t pg_launch_count(void) { return g_pg_launches.load(); }

int32_t pg_ctx_create(int32_t device, void *stream, pg_ctx **out)
{
    PG_REQUIRE(out != nullptr, "pg_ctx_create: out is null");
    *out = nullptr;
    int count = 0;
    cudaError_t e = cudaGetDeviceCount(&count);
    if (e != cudaSuccess || count == 0)
        PG_FAIL(PG_ERR_UNSUPPORTED, "no CUDA device is visible (%s); this library has no CPU path",
                e == cudaSuccess ? "device count 0" : cudaGetErrorString(e));
    PG_REQUIRE(device >= 0 && device < count, "pg_ctx_create: device %d out of range (0..%d)", device, count - 1);
    cudaDeviceProp prop;
    PG_CUDA(cudaGetDeviceProperties(&prop, device));
    if (prop.major != 10)
        PG_FAIL(PG_ERR_UNSUPPORTED, "device %d is sm_%d%d; the kernels are built for sm_100a only", device, prop.major, prop.minor);
    DeviceGuard guard(device);
    if (!guard.ok) PG_FAIL(PG_ERR_CUDA, "cudaSetDevice(%d) failed", device);
    pg_ctx *ctx = new (std::nothrow) pg_ctx();
    if (!ctx) PG_FAIL(PG_ERR_NOMEM, "out of host memory");
    ctx->device = device;
    ctx->sm_count = prop.multiProcessorCount;
    if (stream) {
        ctx->stream = (cudaStream_t)stream;
    } else {
        cudaError_t se = cudaStreamCreateWithFlags(&ctx->stream, cudaStreamNonBlocking);
        if (se != cudaSuccess) {
            delete ctx;
            PG_FAIL(PG_ERR_CUDA, "cudaStreamCreate failed: %s", cudaGetErrorString(se));
        }
        ctx->owns_stream = true;
    }
    cudaError_t me = cudaMalloc(&ctx->d_status, 16 * sizeof(int32_t));  // [0] status word; the rest is spare
    if (me == cudaSuccess) me = cudaMemset(ctx->d_status, 0, 16 * sizeof(int32_t));
    if (me != cudaSuccess) {
        if (ctx->owns_stream) cudaStreamDestroy(ctx->stream);
        delete ctx;
        PG_FAIL(PG_ERR_CUDA, "status word allocation failed: %s", cudaGetErrorString(me));
    }
    *out = ctx;
    return PG_OK;
}

int32_t pg_ctx_destroy(pg_ctx *ctx)
{
    if (!ctx) return PG_OK;
    DeviceGuard guard(ctx->device);
    cudaStreamSynchronize(ctx->stream);
    if (ctx->scratch) cudaFree(ctx->scratch);
    if (ctx->staging) cudaFree(ctx->staging);
    if (ctx->splitk) cudaFree(ctx->splitk);
    for (void *p : ctx->retired) cudaFree(p);
    for (auto &h : ctx->host_calls)
        if (h.exec) cudaGraphExecDestroy(h.exec);
    if (ctx->d_status) cudaFree(ctx->d_status);
    if (ctx->h_pinned) cudaFreeHost(ctx->h_pinned);
    if (ctx->owns_stream) cudaStreamDestroy(ctx->stream);
    delete ctx;
    return PG_OK;
}

int32_t pg_ctx_sync(pg_ctx *ctx)
{
    PG_ENTER(ctx);
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    return PG_OK;
}

void *pg_ctx_stream(pg_ctx *ctx) { return ctx ? (void *)ctx->stream : nullptr; }

int32_t pg_ctx_device_status(pg_ctx *ctx, int32_t *status_out)
{
    PG_ENTER(ctx);
    int32_t v = 0;
    PG_CUDA(cudaMemcpyAsync(&v, ctx->d_status, sizeof(v), cudaMemcpyDeviceToHost, ctx->stream));
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    if (v != 0) {
        PG_CUDA(cudaMemsetAsync(ctx->d_status, 0, sizeof(v), ctx->stream));
        // a kernel that gave up may have left tickets of the split-K workspace taken: back to zero for the next call
        if (ctx->splitk) PG_CUDA(cudaMemsetAsync(ctx->splitk, 0, std::min(ctx->splitk_bytes, (size_t)64 * 1024), ctx->stream));
    }
    if (status_out) *status_out = v;
    return PG_OK;
}

int32_t pg_ctx_set_wait_limit_ns(pg_ctx *ctx, uint64_t ns)
{
    PG_REQUIRE(ctx != nullptr, "null context");
    PG_REQUIRE(ns >= 1000, "pg_ctx_set_wait_limit_ns: a limit below a microsecond would end waits that are about to succeed");
    ctx->wait_limit_ns = ns;
    return PG_OK;
}

uint64_t pg_ctx_scratch_bytes(const pg_ctx *ctx) { return ctx ? (uint64_t)(ctx->scratch_bytes + ctx->staging_bytes + ctx->splitk_bytes) : 0; }

int32_t pg_graph_begin(pg_ctx *ctx)
{
    PG_ENTER(ctx);
    PG_REQUIRE(!ctx->capturing, "pg_graph_begin: already recording");
    PG_CUDA(cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal));
    ctx->capturing = true;
    return PG_OK;
}

int32_t pg_graph_end(pg_ctx *ctx, pg_graph **out)
{
    PG_ENTER(ctx);
    PG_REQUIRE(out != nullptr, "pg_graph_end: out is null");
    *out = nullptr;
    PG_REQUIRE(ctx->capturing, "pg_graph_end: not recording");
    ctx->capturing = false;
    cudaGraph_t g = nullptr;
    // cudaStreamEndCapture ends the capture even when a recorded call had failed and invalidated it
    const cudaError_t ce = cudaStreamEndCapture(ctx->stream, &g);
    if (ce != cudaSuccess || !g) {
        cudaGetLastError();
        if (g) cudaGraphDestroy(g);
        PG_FAIL(PG_ERR_CUDA, "pg_graph_end: the recording was invalidated (%s); nothing was recorded", cudaGetErrorString(ce));
    }
    cudaGraphExec_t exec = nullptr;
    cudaError_t e = cudaGraphInstantiate(&exec, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) PG_FAIL(PG_ERR_CUDA, "cudaGraphInstantiate failed: %s", cudaGetErrorString(e));
    pg_graph *pgg = new (std::nothrow) pg_graph();
    if (!pgg) {
        cudaGraphExecDestroy(exec);
        PG_FAIL(PG_ERR_NOMEM, "out of host memory");
    }
    pgg->exec = exec;
    ctx->live_graphs++;
    *out = pgg;
    return PG_OK;
}

int32_t pg_graph_launch(pg_ctx *ctx, pg_graph *graph)
{
    PG_ENTER(ctx);
    PG_REQUIRE(graph && graph->exec, "pg_graph_launch: graph is null");
    PG_CUDA(cudaGraphLaunch(graph->exec, ctx->stream));
    return PG_OK;
}

int32_t pg_graph_free(pg_ctx *ctx, pg_graph *graph)
{
    if (!graph) return PG_OK;
    PG_ENTER(ctx);
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    if (graph->exec) cudaGraphExecDestroy(graph->exec);
    delete graph;
    if (ctx->live_graphs > 0 && --ctx->live_graphs == 0) {
        for (void *p : ctx->retired) cudaFree(p);
        ctx->retired.clear();
    }
    return PG_OK;
}

int32_t pg_mem_alloc(pg_ctx *ctx, size_t bytes, void **d_out)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_out != nullptr, "pg_mem_alloc: out is null");
    *d_out = nullptr;
    PG_CUDA(cudaMalloc(d_out, bytes ? bytes : 1));
    return PG_OK;
}

int32_t pg_mem_free(pg_ctx *ctx, void *d_ptr)
{
    PG_ENTER(ctx);
    if (d_ptr) {
        PG_CUDA(cudaStreamSynchronize(ctx->stream));
        PG_CUDA(cudaFree(d_ptr));
    }
    return PG_OK;
}

int32_t pg_mem_upload(pg_ctx *ctx, void *d_dst, const void *src, size_t bytes)
{
    PG_ENTER(ctx);
    if (bytes == 0) return PG_OK;
    PG_REQUIRE(d_dst && src, "pg_mem_upload: null pointer");
    PG_CUDA(cudaMemcpyAsync(d_dst, src, bytes, cudaMemcpyHostToDevice, ctx->stream));
    return PG_OK;
}

int32_t pg_mem_download(pg_ctx *ctx, void *dst, const void *d_src, size_t bytes)
{
    PG_ENTER(ctx);
    if (bytes) {
        PG_REQUIRE(dst && d_src, "pg_mem_download: null pointer");
        PG_CUDA(cudaMemcpyAsync(dst, d_src, bytes, cudaMemcpyDeviceToHost, ctx->stream));
    }
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    return PG_OK;
}

}  // extern "C"
