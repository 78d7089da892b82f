// Context management behind the C ABI of include/b200gpt2.h: creation, the stream binding, the device status
// word, status strings and the cache of tensor maps.
#include <cstdlib>
#include "ctx.h"
#include "../kernels/kernels.h"

int b200_fail_cuda(b200_ctx* ctx, cudaError_t e, const char* what) {
    if (ctx) ctx->last_error = std::string(what) + ": " + cudaGetErrorString(e);
    return B200_ERR_CUDA;
}

int b200_get_tensor_map(b200_ctx* ctx, CUtensorMap* out, const float* ptr, uint64_t rows,
                        uint64_t cols, uint64_t ld, uint32_t box_rows, uint32_t box_cols,
                        int swizzle_atom32) {
    TensorMapKey key{ptr, rows, cols, ld, box_rows, box_cols, swizzle_atom32};
    auto it = ctx->tmap_cache.find(key);
    if (it != ctx->tmap_cache.end()) { *out = it->second; return B200_OK; }
    if (!ctx->encode_tiled) return B200_ERR_STATE;
    if (!b200_aligned16(ptr) || (ld * 4) % 16 != 0) return B200_ERR_ALIGN;
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {ld * sizeof(float)};
    const cuuint32_t box[2] = {box_cols, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    CUtensorMap m;
    CUresult r = ctx->encode_tiled(&m, CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 2, const_cast<float*>(ptr), dims,
                                   strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                   swizzle_atom32 ? CU_TENSOR_MAP_SWIZZLE_128B_ATOM_32B : CU_TENSOR_MAP_SWIZZLE_128B,
                                   CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        ctx->last_error = "cuTensorMapEncodeTiled failed with CUresult " + std::to_string((int)r);
        return B200_ERR_CUDA;
    }
    if (ctx->tmap_cache.size() > 4096) ctx->tmap_cache.clear();
    ctx->tmap_cache.emplace(key, m);
    *out = m;
    return B200_OK;
}

int b200_get_tensor_map_bf16(b200_ctx* ctx, CUtensorMap* out, const void* ptr, uint64_t rows,
                             uint64_t cols, uint64_t ld, uint32_t box_rows, uint32_t box_cols) {
    TensorMapKey key{ptr, rows, cols, ld, box_rows, box_cols, 2};  // 2: 16-bit elements
    auto it = ctx->tmap_cache.find(key);
    if (it != ctx->tmap_cache.end()) { *out = it->second; return B200_OK; }
    if (!ctx->encode_tiled) return B200_ERR_STATE;
    if (!b200_aligned16(ptr) || (ld * 2) % 16 != 0) return B200_ERR_ALIGN;
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {ld * 2};
    const cuuint32_t box[2] = {box_cols, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    CUtensorMap m;
    CUresult r = ctx->encode_tiled(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims,
                                   strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                   CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        ctx->last_error = "cuTensorMapEncodeTiled (bf16) failed with CUresult " + std::to_string((int)r);
        return B200_ERR_CUDA;
    }
    if (ctx->tmap_cache.size() > 4096) ctx->tmap_cache.clear();
    ctx->tmap_cache.emplace(key, m);
    *out = m;
    return B200_OK;
}

int b200_get_tensor_map_u8(b200_ctx* ctx, CUtensorMap* out, const void* ptr, uint64_t rows,
                           uint64_t cols, uint64_t ld, uint32_t box_rows, uint32_t box_cols) {
    TensorMapKey key{ptr, rows, cols, ld, box_rows, box_cols, 3};  // 3: 8-bit elements
    auto it = ctx->tmap_cache.find(key);
    if (it != ctx->tmap_cache.end()) { *out = it->second; return B200_OK; }
    if (!ctx->encode_tiled) return B200_ERR_STATE;
    if (!b200_aligned16(ptr) || ld % 16 != 0) return B200_ERR_ALIGN;
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {ld};
    const cuuint32_t box[2] = {box_cols, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    CUtensorMap m;
    CUresult r = ctx->encode_tiled(&m, CU_TENSOR_MAP_DATA_TYPE_UINT8, 2, const_cast<void*>(ptr), dims,
                                   strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                   CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        ctx->last_error = "cuTensorMapEncodeTiled (8-bit) failed with CUresult " + std::to_string((int)r);
        return B200_ERR_CUDA;
    }
    if (ctx->tmap_cache.size() > 4096) ctx->tmap_cache.clear();
    ctx->tmap_cache.emplace(key, m);
    *out = m;
    return B200_OK;
}

extern "C" {

const char* b200_status_string(int s) {
    switch (s) {
        case B200_OK: return "ok";
        case B200_ERR_NULL: return "required pointer is NULL";
        case B200_ERR_SHAPE: return "dimension violates a precondition";
        case B200_ERR_ALIGN: return "pointer is not 16-byte aligned";
        case B200_ERR_CUDA: return "CUDA call failed";
        case B200_ERR_DEVICE: return "device is not sm_100";
        case B200_ERR_TIMEOUT: return "device-side wait ran out";
        case B200_ERR_STATE: return "object not set up";
        case B200_ERR_LIMIT: return "size beyond the stated maximum";
        default: return "unknown status";
    }
}

int b200_ctx_create(b200_ctx** out, int device, void* stream) {
    if (!out) return B200_ERR_NULL;
    *out = nullptr;
    b200_ctx* ctx = new b200_ctx();
    ctx->device = device;
    ctx->stream = static_cast<cudaStream_t>(stream);
    cudaError_t e = cudaSetDevice(device);
    cudaDeviceProp prop;
    if (e == cudaSuccess) e = cudaGetDeviceProperties(&prop, device);
    if (e != cudaSuccess) { delete ctx; return B200_ERR_CUDA; }
    if (prop.major != 10) { delete ctx; return B200_ERR_DEVICE; }
    ctx->num_sms = prop.multiProcessorCount;
    e = cudaMalloc(&ctx->d_status, 256);
    if (e == cudaSuccess) e = cudaMemset(ctx->d_status, 0, 256);
    if (e == cudaSuccess) e = cudaHostAlloc(&ctx->h_status, sizeof(int), cudaHostAllocDefault);
    ctx->split_flag_words = (size_t)1 << 18;  // 1 MB: up to 16384 K-slice tiles per launch
    if (e == cudaSuccess) e = cudaMalloc(&ctx->d_split_flags, ctx->split_flag_words * sizeof(unsigned int));
    if (e == cudaSuccess) e = cudaMemset(ctx->d_split_flags, 0, ctx->split_flag_words * sizeof(unsigned int));
    if (e != cudaSuccess) { cudaFree(ctx->d_status); cudaFree(ctx->d_split_flags); delete ctx; return B200_ERR_CUDA; }
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult qres;
    e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres);
    if (e != cudaSuccess || qres != cudaDriverEntryPointSuccess || !fn) {
        cudaFree(ctx->d_status);
        cudaFree(ctx->d_split_flags);
        cudaFreeHost(ctx->h_status);
        delete ctx;
        return B200_ERR_CUDA;
    }
    ctx->encode_tiled = reinterpret_cast<b200_encode_tiled_fn>(fn);
    if (const char* e = getenv("B200_PDL")) ctx->pdl = !(e[0] == '0');
    *out = ctx;
    return B200_OK;
}

int b200_ctx_destroy(b200_ctx* ctx) {
    if (!ctx) return B200_ERR_NULL;
    cudaSetDevice(ctx->device);
    cudaFree(ctx->d_status);
    cudaFree(ctx->d_split_flags);
    cudaFreeHost(ctx->h_status);
    if (ctx->own_stream) cudaStreamDestroy(ctx->own_stream);
    delete ctx;
    return B200_OK;
}

int b200_ctx_own_stream(b200_ctx* ctx) {
    if (!ctx) return B200_ERR_NULL;
    b200_device_guard guard(ctx);
    if (!ctx->own_stream) B200_CUDA(ctx, cudaStreamCreateWithFlags(&ctx->own_stream, cudaStreamNonBlocking));
    ctx->stream = ctx->own_stream;
    return B200_OK;
}

int b200_ctx_set_stream(b200_ctx* ctx, void* stream) {
    if (!ctx) return B200_ERR_NULL;
    ctx->stream = static_cast<cudaStream_t>(stream);
    return B200_OK;
}

int b200_ctx_sync_check(b200_ctx* ctx) {
    if (!ctx) return B200_ERR_NULL;
    // the status word rides behind the queued work: one wait for both
    B200_CUDA(ctx, cudaMemcpyAsync(ctx->h_status, ctx->d_status, sizeof(int), cudaMemcpyDeviceToHost, ctx->stream));
    B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    const int word = *ctx->h_status;
    if (word != 0) {
        // the whole area: a kernel that gave up may have left its work counters behind (and a GEMM
        // with K slices its hand-over flags)
        B200_CUDA(ctx, cudaMemset(ctx->d_status, 0, 256));
        B200_CUDA(ctx, cudaMemset(ctx->d_split_flags, 0, ctx->split_flag_words * sizeof(unsigned int)));
        ctx->last_error = "device status word = " + std::to_string(word);
        return word == 201 ? B200_ERR_SHAPE : B200_ERR_TIMEOUT;
    }
    B200_CUDA(ctx, cudaGetLastError());
    return B200_OK;
}

int b200_ctx_wait_timeout_probe(b200_ctx* ctx, int limit_ms) {
    if (!ctx) return B200_ERR_NULL;
    if (limit_ms < 1 || limit_ms > 2000) return B200_ERR_SHAPE;
    return b200::launch_wait_timeout_probe(ctx, (unsigned long long)limit_ms * 1000000ull);
}

int b200_ctx_peer_wait_probe(b200_ctx* ctx, int limit_ms) {
    if (!ctx) return B200_ERR_NULL;
    if (limit_ms < 1 || limit_ms > 2000) return B200_ERR_SHAPE;
    // word 40 of the status area is never written: the wait for it to reach 1 runs out
    return b200::launch_peer_wait(ctx, reinterpret_cast<const unsigned int*>(ctx->d_status + 40), 1u, (unsigned long long)limit_ms * 1000000ull);
}

// debugging aid for kernel experiments: device address of the status words
void* b200_ctx_debug_status(b200_ctx* ctx) { return ctx ? ctx->d_status : nullptr; }

uint64_t b200_ctx_launch_count(const b200_ctx* ctx) { return ctx ? ctx->launches : 0; }
void b200_ctx_reset_launch_count(b200_ctx* ctx) { if (ctx) ctx->launches = 0; }
const char* b200_ctx_last_error(const b200_ctx* ctx) { return ctx ? ctx->last_error.c_str() : ""; }

}  // extern "C"
