// Memory-bound kernels of the step: embedding gather, residual add fused with RMSNorm,
// per-head q/k RMSNorm fused with rotary position encoding and the cache write, and the
// SiLU-gated product.  Norms, rotation and the residual sum are computed in float.
//
// Counterparts in luozoupi/Qwen-Triton: kernels/embedding.py:50-66, kernels/rmsnorm.py:100-133,
// kernels/residual_add.py:50-60, kernels/rope.py:99-120, csrc/rope_op_kernel.cu:12-39,
// kernels/cache.py:71-98, kernels/swiglu.py:84-92.
#include "common.cuh"

using namespace qt;

// ----------------------------------------------------------------------------- embedding
// residual[t, c, :] = table[ids[t], :] widened to float, times `scale` (1 for a plain gather), for every c of `copies` (a residual
// of several parallel streams starts with all of them alike; 1: the plain stream).  One block per token.
template <typename T>
__global__ void embedding_kernel(float* __restrict__ residual, const T* __restrict__ table,
                                 const int* __restrict__ ids, int hidden, int vocab, float scale, int copies) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int id = ids[t];
    const bool valid = id >= 0 && id < vocab;   // ids are range-checked on the host; never read outside the table
    const T* row = table + (size_t)(valid ? id : 0) * hidden;
    float* out = residual + (size_t)t * copies * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float x = valid ? to_float(row[i]) * scale : 0.f;
        for (int c = 0; c < copies; ++c) out[(size_t)c * hidden + i] = x;
    }
}

// The same with an RMS norm behind the gather: residual[t, :] = x / sqrt(mean(x^2) + eps) * norm_w for the scaled row x.
// `start` (or null) takes a copy of the result in the table's type: the embedding's output, for a model whose layers
// meet it again.  One block per token.
template <typename T>
__global__ void embedding_norm_kernel(float* __restrict__ residual, const T* __restrict__ table, const int* __restrict__ ids, int hidden,
                                      int vocab, float scale, const float* __restrict__ norm_w, float eps, T* __restrict__ start) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    int id = ids[t];
    const bool valid = id >= 0 && id < vocab;
    const T* row = table + (size_t)(valid ? id : 0) * hidden;
    constexpr int KEEP = 16;                                  // elements a thread keeps; wider rows are read again
    float x[KEEP], sq = 0.f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        x[j] = i < hidden && valid ? to_float(row[i]) * scale : 0.f;
        sq += x[j] * x[j];
    }
    for (int i = threadIdx.x + KEEP * blockDim.x; i < hidden; i += blockDim.x) { const float v = valid ? to_float(row[i]) * scale : 0.f; sq += v * v; }
    const float inv = norm_w ? rsqrtf(block_sum(sq, scratch) / (float)hidden + eps) : 1.f;
    auto put = [&](int i, float v) {
        const float y = v * inv * (norm_w ? __ldg(norm_w + i) : 1.f);
        residual[(size_t)t * hidden + i] = y;
        if (start) start[(size_t)t * hidden + i] = from_float<T>(y);
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j)
        if (threadIdx.x + j * blockDim.x < hidden) put(threadIdx.x + j * blockDim.x, x[j]);
    for (int i = threadIdx.x + KEEP * blockDim.x; i < hidden; i += blockDim.x) put(i, valid ? to_float(row[i]) * scale : 0.f);
}

extern "C" int qt_embedding(float* residual, const void* table, const int* ids, int n_tokens, int hidden, int vocab,
                            int table_dtype, float scale, const float* norm_w, float eps, void* start, int copies, void* stream) {
    QT_REQUIRE(copies >= 1 && (copies == 1 || (!norm_w && !start)), "embedding: %d copies of a row that is normed or kept", copies);
    QT_REQUIRE(n_tokens >= 0 && hidden > 0 && vocab > 0, "embedding: bad sizes T=%d H=%d V=%d", n_tokens, hidden, vocab);
    QT_REQUIRE(!norm_w || eps > 0.f, "embedding: eps must be positive");
    if (n_tokens == 0) return QT_OK;
    return QT_DISPATCH_DTYPE(table_dtype, "embedding", {
        if (norm_w || start) {
            launch_kernel(embedding_norm_kernel<T>, dim3(n_tokens), dim3(256), 0, (cudaStream_t)stream, residual, (const T*)table, ids, hidden, vocab, scale,
                          norm_w, eps, (T*)start);
            QT_CHECK_LAUNCH("embedding_norm");
            return QT_OK;
        }
        launch_kernel(embedding_kernel<T>, dim3(n_tokens), dim3(256), 0, (cudaStream_t)stream, residual, (const T*)table, ids, hidden, vocab, scale, copies);
        QT_CHECK_LAUNCH("embedding");
        return QT_OK;
    });
}

// ----------------------------------------------------------------------------- the stream beside the embedding's output
// out[t] = [x | start[t]] in the activation type, x = residual[t] + sum_s delta[s][t] in float; the stream is then zero:
// what a map of these rows returns takes its place by the ordinary addition of the next norm.  One block per token.
template <typename TD, typename TO>
__global__ void stream_concat_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_splits, size_t split_stride,
                                     const TO* __restrict__ start, TO* __restrict__ out, int hidden) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t at = (size_t)blockIdx.x * hidden, to = 2 * at;
    constexpr int AHEAD = 8;                                  // elements a thread asks for before it stores the first
    for (int i0 = threadIdx.x; i0 < hidden; i0 += AHEAD * blockDim.x) {
        float x[AHEAD];
        TO s[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int i = i0 + j * blockDim.x;
            x[j] = 0.f;
            if (i < hidden) {
                x[j] = residual[at + i];
                s[j] = start[at + i];
                if (delta) x[j] += load_sum(delta, at + i, n_splits, split_stride);
            }
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int i = i0 + j * blockDim.x;
            if (i >= hidden) break;
            residual[at + i] = 0.f;
            out[to + i] = from_float<TO>(x[j]);
            out[to + hidden + i] = s[j];
        }
    }
}

extern "C" int qt_stream_concat(float* residual, const void* delta, int delta_dtype, int n_splits, long long split_stride, const void* start,
                                void* out, int dtype, int n_tokens, int hidden, void* stream) {
    QT_REQUIRE(n_tokens >= 0 && hidden > 0 && n_splits >= 1, "stream_concat: bad sizes T=%d H=%d splits=%d", n_tokens, hidden, n_splits);
    if (n_tokens == 0) return QT_OK;
    cudaStream_t s = (cudaStream_t)stream;
#define QT_LAUNCH_CONCAT(TD, TO)                                                                                                  \
    launch_kernel(stream_concat_kernel<TD, TO>, dim3(n_tokens), dim3(256), 0, s, residual, (const TD*)delta, n_splits, (size_t)split_stride, \
                  (const TO*)start, (TO*)out, hidden)
    if (delta_dtype == QT_F32 && dtype == QT_F32) QT_LAUNCH_CONCAT(float, float);
    else if (delta_dtype == QT_F32 && dtype == QT_BF16) QT_LAUNCH_CONCAT(float, __nv_bfloat16);
    else if (delta_dtype == QT_BF16 && dtype == QT_BF16) QT_LAUNCH_CONCAT(__nv_bfloat16, __nv_bfloat16);
    else QT_FAIL(QT_ERR_ARG, "stream_concat: element types %d/%d", delta_dtype, dtype);
#undef QT_LAUNCH_CONCAT
    QT_CHECK_LAUNCH("stream_concat");
    return QT_OK;
}

// ----------------------------------------------------------------------------- bias of a projection
// out[t, :] += bias, on the float sums of a product before anything rounds them (the first plane, where a product is
// split over K).  luozoupi/Qwen-Triton adds the bias of a linear layer with a kernel of its own as well
// (kernels/matmul.py:99-111, modules/linear.py:31).
__global__ void add_bias_kernel(float* __restrict__ out, const float* __restrict__ bias, int cols, size_t count) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x)
        out[i] += bias[i % (size_t)cols];
}

extern "C" int qt_add_bias(float* out, const float* bias, int rows, int cols, void* stream) {
    QT_REQUIRE(rows >= 0 && cols > 0, "add_bias: bad sizes rows=%d cols=%d", rows, cols);
    if (rows == 0) return QT_OK;
    const size_t count = (size_t)rows * cols;
    const size_t blocks = (count + 255) / 256;
    launch_kernel(add_bias_kernel, dim3((unsigned)(blocks < 4096 ? blocks : 4096)), dim3(256), 0, (cudaStream_t)stream, out, bias, cols, count);
    QT_CHECK_LAUNCH("add_bias");
    return QT_OK;
}

// ----------------------------------------------------------------------------- residual add + RMSNorm
// One block per output row r.  src = rows ? rows[r] : r.
//   x = residual[src] + sum_s delta[s][src]            (float)
//   if (!rows) residual[src] = x                        (the stream is updated in place)
//   out[r] = x * rsqrt(mean(x^2) + eps) * weight       (rounded once to the output type)
// With `rows` the kernel norms only the listed rows (the positions whose logits are wanted) and
// leaves the stream untouched.
// Norm in groups: a row of `width` elements is `gridDim.y` equal consecutive parts of `hidden` elements, each
// divided by its own root mean square (blockIdx.y is the part); one part is the plain norm.
template <typename TD, typename TO>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_splits,
                                   size_t split_stride, const float* __restrict__ weight, float eps,
                                   TO* __restrict__ out, const int* __restrict__ rows, int hidden, int width) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    const size_t part = (size_t)blockIdx.y * hidden;
    float* res = residual + (size_t)src * width + part;
    if (delta) delta += part;
    weight += part;
    out += part;
    float sq = 0.f;
    // pass 1: form the new stream value; keep it in `res` (or, for listed rows, recompute in pass 2)
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float x = res[i];
        if (delta) x += load_sum(delta, (size_t)src * width + i, n_splits, split_stride);
        if (!rows) res[i] = x;
        sq += x * x;
    }
    const float total = block_sum(sq, scratch);
    const float inv = rsqrtf(total / (float)hidden + eps);
    TO* o = out + (size_t)r * width;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float x = res[i];   // each thread re-reads what it wrote itself
        if (rows && delta) x += load_sum(delta, (size_t)src * width + i, n_splits, split_stride);
        o[i] = from_float<TO>(x * inv * weight[i]);
    }
}

// Vector form for widths that are multiples of 4: each thread owns up to NORM_CACHE chunks of four
// consecutive elements, sums the split-K partials with independent 16-byte loads and keeps the new
// stream values in registers between the two passes.
constexpr int NORM_CACHE = 4;

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&a);
    raw.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// v += sum over splits of the four elements at dp + s * split_stride, in the order of the splits.  Up to sixteen
// loads are issued before the first add: with one block per few hundred elements the kernel's time is the chain of
// L2 round trips, not the bytes.
template <int BATCH, typename TD>
__device__ __forceinline__ void add_splits4(float4& v, const TD* dp, int first, int n_splits, size_t split_stride) {
    for (int s0 = first; s0 < n_splits; s0 += BATCH) {
        float4 t[BATCH];
#pragma unroll
        for (int j = 0; j < BATCH; ++j)               // unconditional loads (the last split again beyond the end), so that they batch
            t[j] = load4(dp + (size_t)min(s0 + j, n_splits - 1) * split_stride);
#pragma unroll
        for (int j = 0; j < BATCH; ++j)
            if (s0 + j < n_splits) { v.x += t[j].x; v.y += t[j].y; v.z += t[j].z; v.w += t[j].w; }
    }
}

template <typename TD, typename TO, int BATCH, int MAX_THREADS, int MIN_BLOCKS>
__global__ void __launch_bounds__(MAX_THREADS, MIN_BLOCKS) add_rmsnorm_vec_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_splits,
                                       size_t split_stride, const float* __restrict__ weight, float eps,
                                       TO* __restrict__ out, const int* __restrict__ rows, int hidden, int width) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    const size_t part = (size_t)blockIdx.y * hidden;          // norm in groups: see add_rmsnorm_kernel
    float* res = residual + (size_t)src * width + part;
    if (delta) delta += part;
    weight += part;
    out += part;
    const int chunks = hidden >> 2;
    float4 x[NORM_CACHE];
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < NORM_CACHE; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
            float4 v = load4(res + 4 * c);
            if (delta) add_splits4<BATCH>(v, delta + (size_t)src * width + 4 * c, 0, n_splits, split_stride);
            if (!rows) store4(res + 4 * c, v);
            x[i] = v;
            sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    }
    const float total = block_sum(sq, scratch);
    const float inv = rsqrtf(total / (float)hidden + eps);
    TO* o = out + (size_t)r * width;
#pragma unroll
    for (int i = 0; i < NORM_CACHE; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
            const float4 w = load4(weight + 4 * c);
            store4(o + 4 * c, make_float4(x[i].x * inv * w.x, x[i].y * inv * w.y, x[i].z * inv * w.z, x[i].w * inv * w.w));
        }
    }
}

// Few rows (a decode step): a cluster of NORM_CLUSTER blocks per row, one chunk of four elements per thread, so that
// 8 rows keep 64 SMs busy instead of 8.  Each block pushes its share of the sum of squares into every block of its
// cluster (distributed shared memory); after the cluster barrier each block adds the shares up in the same order.
constexpr int NORM_CLUSTER = 8;

template <typename TD, typename TO>
__global__ void __launch_bounds__(1024, 1) add_rmsnorm_cluster_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_splits,
                                                                   size_t split_stride, const float* __restrict__ weight, float eps,
                                                                   TO* __restrict__ out, const int* __restrict__ rows, int hidden) {
    pdl_launch_dependents();
    cluster_arrive_started();
    pdl_wait();
    __shared__ float scratch[32];
    __shared__ float shares[NORM_CLUSTER];
    const uint32_t rank = cluster_rank();
    const int r = blockIdx.x / NORM_CLUSTER;
    const int src = rows ? rows[r] : r;
    float* res = residual + (size_t)src * hidden;
    const int chunks = hidden >> 2;
    const int c = (int)rank * blockDim.x + threadIdx.x;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < chunks) {
        v = load4(res + 4 * c);
        if (delta) add_splits4<16>(v, delta + (size_t)src * hidden + 4 * c, 0, n_splits, split_stride);
        if (!rows) store4(res + 4 * c, v);
    }
    const float4 w = c < chunks ? load4(weight + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);   // in flight under the reductions
    const float share = block_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w, scratch);
    cluster_wait_started();                                    // every block of the cluster runs: its shared memory may be written
    if (threadIdx.x < NORM_CLUSTER) cluster_store_float(&shares[rank], threadIdx.x, share);
    cluster_barrier();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < NORM_CLUSTER; ++i) total += shares[i];
    const float inv = rsqrtf(total / (float)hidden + eps);
    if (c < chunks) {
        store4(out + (size_t)r * hidden + 4 * c, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
    }
}

extern "C" int qt_add_rmsnorm(float* residual, const void* delta, int delta_dtype, int n_splits, long long split_stride,
                              const float* weight, float eps, void* out, int out_dtype, const int* rows, int n_rows,
                              int width, int groups, void* stream) {
    QT_REQUIRE(n_rows >= 0 && width > 0 && n_splits >= 1, "add_rmsnorm: bad sizes rows=%d H=%d splits=%d", n_rows, width, n_splits);
    QT_REQUIRE(groups >= 1 && groups <= 65535 && width % groups == 0, "add_rmsnorm: %d groups do not divide a width of %d", groups, width);
    QT_REQUIRE(eps > 0.f, "add_rmsnorm: eps must be positive");
    if (n_rows == 0) return QT_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int hidden = width / groups;          // elements that share a root mean square
    // the vector kernel needs 16-byte aligned rows everywhere and at most NORM_CACHE chunks per thread
    const bool aligned = hidden % 4 == 0 && ((uintptr_t)residual % 16 == 0) && ((uintptr_t)out % 16 == 0) &&
                         ((uintptr_t)weight % 16 == 0) && (!delta || ((uintptr_t)delta % 16 == 0 && split_stride % 4 == 0));
    if (aligned && groups == 1 && n_rows < 256 && hidden >= 4 * 32 * NORM_CLUSTER && hidden <= 4 * 1024 * NORM_CLUSTER) {
        const int per_block = (hidden / 4 + NORM_CLUSTER - 1) / NORM_CLUSTER;
        const int cthreads = ((per_block + 31) / 32) * 32;
#define QT_LAUNCH_NORM_CLUSTER(TD, TO)                                                                                  \
    launch_kernel_cluster(add_rmsnorm_cluster_kernel<TD, TO>, dim3(n_rows * NORM_CLUSTER), dim3(cthreads), 0, s, NORM_CLUSTER, residual, \
                          (const TD*)delta, n_splits, (size_t)split_stride, weight, eps, (TO*)out, rows, hidden)
        if (delta_dtype == QT_F32 && out_dtype == QT_F32) QT_LAUNCH_NORM_CLUSTER(float, float);
        else if (delta_dtype == QT_F32 && out_dtype == QT_BF16) QT_LAUNCH_NORM_CLUSTER(float, __nv_bfloat16);
        else if (delta_dtype == QT_BF16 && out_dtype == QT_BF16) QT_LAUNCH_NORM_CLUSTER(__nv_bfloat16, __nv_bfloat16);
        else if (delta_dtype == QT_BF16 && out_dtype == QT_F32) QT_LAUNCH_NORM_CLUSTER(__nv_bfloat16, float);
        else QT_FAIL(QT_ERR_ARG, "add_rmsnorm: unknown element types %d/%d", delta_dtype, out_dtype);
#undef QT_LAUNCH_NORM_CLUSTER
        QT_CHECK_LAUNCH("add_rmsnorm");
        return QT_OK;
    }
    if (aligned && hidden <= 4 * NORM_CACHE * 1024) {
        // few rows (decode): one chunk per thread, shortest critical path; many rows (prefill): up to NORM_CACHE
        // independent chunks per thread in smaller blocks, which keeps more loads in flight and more blocks resident
        const int per_thread = n_rows >= 256 ? NORM_CACHE : 1;
        int vthreads = ((hidden / 4 + 32 * per_thread - 1) / (32 * per_thread)) * 32;
        if (vthreads > 1024) vthreads = 1024;
        if (vthreads < 64) vthreads = 64;
        // many rows in blocks of up to 256 threads: few registers, five blocks per SM (partial sums of a split product
        // are rare there); otherwise up to 1,024 threads with eight loads of partial sums in flight
#define QT_NORM_VEC_ARGS residual, (const TD_*)delta, n_splits, (size_t)split_stride, weight, eps, (TO_*)out, rows, hidden, width
#define QT_LAUNCH_NORM_VEC(TD, TO)                                                                                      \
    do {                                                                                                                \
        using TD_ = TD; using TO_ = TO;                                                                                 \
        if (per_thread > 1 && vthreads <= 256)                                                                          \
            launch_kernel(add_rmsnorm_vec_kernel<TD, TO, 2, 256, 5>, dim3(n_rows, groups), dim3(vthreads), 0, s, QT_NORM_VEC_ARGS); \
        else                                                                                                            \
            launch_kernel(add_rmsnorm_vec_kernel<TD, TO, 8, 1024, 1>, dim3(n_rows, groups), dim3(vthreads), 0, s, QT_NORM_VEC_ARGS); \
    } while (0)
        if (delta_dtype == QT_F32 && out_dtype == QT_F32) QT_LAUNCH_NORM_VEC(float, float);
        else if (delta_dtype == QT_F32 && out_dtype == QT_BF16) QT_LAUNCH_NORM_VEC(float, __nv_bfloat16);
        else if (delta_dtype == QT_BF16 && out_dtype == QT_BF16) QT_LAUNCH_NORM_VEC(__nv_bfloat16, __nv_bfloat16);
        else if (delta_dtype == QT_BF16 && out_dtype == QT_F32) QT_LAUNCH_NORM_VEC(__nv_bfloat16, float);
        else QT_FAIL(QT_ERR_ARG, "add_rmsnorm: unknown element types %d/%d", delta_dtype, out_dtype);
#undef QT_LAUNCH_NORM_VEC
#undef QT_NORM_VEC_ARGS
        QT_CHECK_LAUNCH("add_rmsnorm");
        return QT_OK;
    }
    const int threads = hidden >= 2048 ? 512 : 256;
#define QT_LAUNCH_NORM(TD, TO)                                                                                   \
    launch_kernel(add_rmsnorm_kernel<TD, TO>, dim3(n_rows, groups), dim3(threads), 0, s, residual, (const TD*)delta, n_splits, (size_t)split_stride, \
                                                          weight, eps, (TO*)out, rows, hidden, width)
    if (delta_dtype == QT_F32 && out_dtype == QT_F32) QT_LAUNCH_NORM(float, float);
    else if (delta_dtype == QT_F32 && out_dtype == QT_BF16) QT_LAUNCH_NORM(float, __nv_bfloat16);
    else if (delta_dtype == QT_BF16 && out_dtype == QT_BF16) QT_LAUNCH_NORM(__nv_bfloat16, __nv_bfloat16);
    else if (delta_dtype == QT_BF16 && out_dtype == QT_F32) QT_LAUNCH_NORM(__nv_bfloat16, float);
    else QT_FAIL(QT_ERR_ARG, "add_rmsnorm: unknown element types %d/%d", delta_dtype, out_dtype);
#undef QT_LAUNCH_NORM
    QT_CHECK_LAUNCH("add_rmsnorm");
    return QT_OK;
}

// ----------------------------------------------------------------------------- residual add + Dynamic Tanh
// A norm without statistics: out = tanh(alpha x) * weight + bias, elementwise, alpha one number.  Like the RMSNorm
// kernels it first folds what is pending into the float stream, here up to two additions (a block whose mixer and
// feed-forward read the same normed rows adds both results at once), each possibly split-K partial sums in float:
//   x = residual[src] + sum_s delta_a[s][src] + sum_s delta_b[s][src];  if (!rows) residual[src] = x.
struct DytParams {
    float* residual;
    const float* delta_a; int splits_a; size_t stride_a;
    const float* delta_b; int splits_b; size_t stride_b;
    const float* weight; const float* bias; float alpha;
    void* out; const int* rows; int n_rows, hidden;
};

template <typename TO>
__global__ void add_dyt_kernel(const DytParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const long long total = (long long)p.n_rows * p.hidden;
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const int r = (int)(idx / p.hidden), i = (int)(idx % p.hidden);
        const size_t at = (size_t)(p.rows ? p.rows[r] : r) * p.hidden + i;
        float x = p.residual[at];
        if (p.delta_a) x += load_sum(p.delta_a, at, p.splits_a, p.stride_a);
        if (p.delta_b) x += load_sum(p.delta_b, at, p.splits_b, p.stride_b);
        if (!p.rows) p.residual[at] = x;
        ((TO*)p.out)[idx] = from_float<TO>(tanhf(p.alpha * x) * p.weight[i] + p.bias[i]);
    }
}

extern "C" int qt_add_dyt(float* residual, const float* delta_a, int splits_a, long long stride_a, const float* delta_b, int splits_b,
                          long long stride_b, const float* weight, const float* bias, float alpha, void* out, int out_dtype,
                          const int* rows, int n_rows, int hidden, void* stream) {
    QT_REQUIRE(n_rows >= 0 && hidden > 0 && splits_a >= 1 && splits_b >= 1, "add_dyt: bad sizes rows=%d H=%d", n_rows, hidden);
    if (n_rows == 0) return QT_OK;
    DytParams p{residual, delta_a, splits_a, (size_t)stride_a, delta_b, splits_b, (size_t)stride_b, weight, bias, alpha, out, rows, n_rows, hidden};
    cudaStream_t s = (cudaStream_t)stream;
    const long long total = (long long)n_rows * hidden;
    long long blocks = (total + 255) / 256;
    if (blocks > (long long)sm_count() * 16) blocks = (long long)sm_count() * 16;
    return QT_DISPATCH_DTYPE(out_dtype, "add_dyt", {
        launch_kernel(add_dyt_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, s, p);
        QT_CHECK_LAUNCH("add_dyt");
        return QT_OK;
    });
}

// ----------------------------------------------------------------------------- two attention maps into one head
// Differential attention: a head has two softmax maps over the same values; ctx holds their results as heads
// [map][head] (map-major), and the head's output is o = a1 - lambda * a2, divided by its root mean square over the
// head's values (no weight), times `post`.  One warp per (token, head), float inside.
template <typename T>
__global__ void __launch_bounds__(128) map_difference_kernel(const T* __restrict__ ctx, T* __restrict__ out, long long tokens, int heads,
                                                             int dv, float lambda, float eps, float post) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= tokens * heads) return;
    const long long t = item / heads;
    const int h = (int)(item % heads);
    const T* a1 = ctx + ((size_t)t * 2 * heads + h) * dv;
    const T* a2 = a1 + (size_t)heads * dv;
    float sq = 0.f;
    for (int i = lane; i < dv; i += 32) { const float o = to_float(a1[i]) - lambda * to_float(a2[i]); sq += o * o; }
    const float inv = rsqrtf(warp_sum(sq) / (float)dv + eps) * post;
    for (int i = lane; i < dv; i += 32) out[item * dv + i] = from_float<T>((to_float(a1[i]) - lambda * to_float(a2[i])) * inv);
}

extern "C" int qt_map_difference(const void* ctx, void* out, int dtype, int n_tokens, int heads, int dv, float lambda, float eps,
                                 float post, void* stream) {
    QT_REQUIRE(n_tokens >= 0 && heads > 0 && dv > 0, "map_difference: bad sizes");
    if (n_tokens == 0) return QT_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const long long items = (long long)n_tokens * heads;
    return QT_DISPATCH_DTYPE(dtype, "map_difference", {
        launch_kernel(map_difference_kernel<T>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, s, (const T*)ctx, (T*)out, (long long)n_tokens,
                      heads, dv, lambda, eps, post);
        QT_CHECK_LAUNCH("map_difference");
        return QT_OK;
    });
}

// ----------------------------------------------------------------------------- q/k norm + rotary + cache write
// Input: the fused projection output qkv[t, (nq + 2 nkv) * d] (possibly split-K partial sums).
// One warp per (token, head):
//   q head:  RMSNorm over d with q_weight (if given), rotate, store to q_out[t, h, :]
//   k head:  RMSNorm with k_weight (if given), rotate, store into the key cache at the token's position
//   v head:  store into the value cache
// Rotation: the first rd dims are paired (i, i + rd/2) (rotate-half) or, with `interleaved`, (2i, 2i + 1); pair i
// turns by the angle whose cos/sin come from the float table cos_sin[pos, i] = cos, [pos, rd/2 + i] = sin.
// rd = 0 means no position encoding.
// With kv_in_proj = 0 the projection holds query heads only; with write_kv = 0 the k and v heads
// are skipped (a call that reads the cache another call wrote).
struct QkvParams {
    const void* qkv; int n_splits; size_t split_stride;
    void* q_out; void* k_cache; void* v_cache;
    const int* token_seq; const int* token_pos; const int* block_table; int max_blocks;
    const float* q_weight; const float* k_weight; float eps;
    const float* cos_sin; int rotary_dim; int max_pos;
    int n_tokens, nq, nkv, d, page_tokens, ring_tokens, write_kv, kv_in_proj;
    int interleaved;        // rotation pairs are (2i, 2i + 1) instead of (i, i + rd/2)
    int nv, dv;             // value heads and their size (the keys' unless given)
    int unit_norm;          // q and k heads are divided by their root mean square without a weight
    const float* row_inv;   // [T, 2]: q and k are normed over the whole row of heads with these factors (q_weight [nq d], k_weight [nkv d])
    int extra_cols;         // columns of the projection behind q, k and v that this kernel leaves alone
};

// The factors of a norm over the whole projection: row_inv[t] = {rsqrt(mean(q_t^2) + eps), rsqrt(mean(k_t^2) + eps)} over all
// nq d (nkv d) elements of token t at once.  One block per token.
template <typename TI>
__global__ void qk_row_rms_kernel(const TI* __restrict__ qkv, int n_splits, size_t split_stride, size_t cols, int q_cols, int k_cols, float eps,
                                  float* __restrict__ row_inv) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < q_cols + k_cols; i += blockDim.x) {
        const float x = load_sum(qkv, (size_t)t * cols + i, n_splits, split_stride);
        if (i < q_cols) sq += x * x; else sk += x * x;
    }
    sq = block_sum(sq, scratch);
    sk = block_sum(sk, scratch);
    if (threadIdx.x == 0) {
        row_inv[2 * t] = rsqrtf(sq / (float)q_cols + eps);
        row_inv[2 * t + 1] = k_cols > 0 ? rsqrtf(sk / (float)k_cols + eps) : 0.f;
    }
}

template <typename TI, typename TO, bool VEC>
__global__ void qk_norm_rope_write_kernel(const QkvParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int heads_total = p.nq + (p.kv_in_proj ? p.nkv + p.nv : 0);
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= (long long)p.n_tokens * heads_total) return;
    const int t = (int)(item / heads_total);
    const int head = (int)(item % heads_total);
    const bool is_q = head < p.nq, is_k = !is_q && head < p.nq + p.nkv;
    if (!is_q && !p.write_kv) return;
    if (!is_q && !is_k && (p.nv != p.nkv || p.dv != p.d)) {
        // a value head of its own size: summed, stored
        const int vh = head - p.nq - p.nkv;
        const size_t cols = (size_t)(p.nq + p.nkv) * p.d + (size_t)p.nv * p.dv + (size_t)p.extra_cols;
        const size_t from = (size_t)t * cols + (size_t)(p.nq + p.nkv) * p.d + (size_t)vh * p.dv;
        const int* table = p.block_table + (size_t)p.token_seq[t] * p.max_blocks;
        TO* dst = (TO*)p.v_cache + cache_offset(table, p.token_pos[t], p.ring_tokens, p.page_tokens, p.nv, vh, p.dv);
        const TI* src = (const TI*)p.qkv;
        for (int i0 = lane; i0 < p.dv; i0 += 128) {                 // four elements' loads ahead of their stores
            float v[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) v[j] = i0 + 32 * j < p.dv ? load_sum(src, from + i0 + 32 * j, p.n_splits, p.split_stride) : 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (i0 + 32 * j < p.dv) dst[i0 + 32 * j] = from_float<TO>(v[j]);
        }
        return;
    }
    float* vec = smem + warp * p.d;
    const size_t in_base = (size_t)t * ((size_t)p.nq * p.d + (p.kv_in_proj ? (size_t)p.nkv * p.d + (size_t)p.nv * p.dv : 0) + (size_t)p.extra_cols) +
                           (size_t)head * p.d;
    const TI* in = (const TI*)p.qkv;
    const float* w = is_q ? p.q_weight : (is_k ? p.k_weight : nullptr);
    if (w && p.row_inv) w += (size_t)(is_q ? head : head - p.nq) * p.d;        // a weight over the whole row of heads
    // a rotation leaves a head's sum of squares as it is, so a norm without a weight that follows the rotation has the
    // factor of the sums as they come, and, both being linear, norm and rotation may change places
    const bool normed = (is_q || is_k) && (w || p.unit_norm || p.row_inv);

    // 1. the head's vector in float (split-K partials added up), its sum of squares
    float sq = 0.f;
    if (VEC) {
        for (int c = lane; c < (p.d >> 2); c += 32) {
            float4 v = load4(in + in_base + 4 * c);
            add_splits4<16>(v, in + in_base + 4 * c, 1, p.n_splits, p.split_stride);
            *reinterpret_cast<float4*>(vec + 4 * c) = v;
            sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = lane; i < p.d; i += 32) {
            const float x = load_sum(in, in_base + i, p.n_splits, p.split_stride);
            vec[i] = x;
            sq += x * x;
        }
    }
    // 2. RMSNorm over the head (q and k heads with a weight)
    float inv = 1.f;
    if (normed) inv = p.row_inv ? p.row_inv[2 * t + (is_q ? 0 : 1)] : rsqrtf(warp_sum(sq) / (float)p.d + p.eps);
    __syncwarp();

    TO* dst;
    const int pos = p.token_pos[t];
    if (is_q) {
        dst = (TO*)p.q_out + ((size_t)t * p.nq + head) * p.d;
    } else {
        const int kvh = is_k ? head - p.nq : head - p.nq - p.nkv;
        const int* table = p.block_table + (size_t)p.token_seq[t] * p.max_blocks;
        dst = (TO*)(is_k ? p.k_cache : p.v_cache) + cache_offset(table, pos, p.ring_tokens, p.page_tokens, p.nkv, kvh, p.d);
    }
    // 3. rotate-half over the first rotary_dim dims with the normed values, store
    const int half = p.rotary_dim >> 1;
    const bool rotate = (is_q || is_k) && half > 0;
    const float* cs = p.cos_sin + (size_t)(pos < p.max_pos ? pos : p.max_pos - 1) * p.rotary_dim;
    auto value = [&](int i) { return normed ? (w ? vec[i] * inv * w[i] : vec[i] * inv) : vec[i]; };
    auto rotated = [&](int i) {
        float y = value(i);
        if (rotate && i < p.rotary_dim) {
            if (p.interleaved) {
                const int j = i >> 1;
                y = (i & 1) ? y * cs[j] + value(i - 1) * cs[half + j] : y * cs[j] - value(i + 1) * cs[half + j];
            } else if (i < half) y = y * cs[i] - value(i + half) * cs[half + i];
            else y = y * cs[i - half] + value(i - half) * cs[i];
        }
        return y;
    };
    if (VEC) {
        for (int c = lane; c < (p.d >> 2); c += 32)
            store4(dst + 4 * c, make_float4(rotated(4 * c), rotated(4 * c + 1), rotated(4 * c + 2), rotated(4 * c + 3)));
    } else {
        for (int i = lane; i < p.d; i += 32) dst[i] = from_float<TO>(rotated(i));
    }
}

// Fast form for many tokens: every dimension rotates (rotary_dim == d) and half a head is IT * 32 * E elements, so
// a lane holds the E-element pieces (j, j + d/2) of a rotation pair in registers and nothing passes through shared
// memory.  One warp takes HEADS_PER_WARP consecutive heads of one token, so that position, page and cos/sin are
// looked up once.  Same arithmetic as the kernel above: float norm, weight, then rotation.
constexpr int HEADS_PER_WARP = 4;

template <int E> struct Piece;
template <> struct Piece<1> { float v[1]; };
template <> struct Piece<2> { float v[2]; };

template <int E> __device__ __forceinline__ Piece<E> load_piece(const float* p) {
    Piece<E> r;
    if (E == 2) { const float2 t = *reinterpret_cast<const float2*>(p); r.v[0] = t.x; r.v[E - 1] = t.y; }
    else r.v[0] = p[0];
    return r;
}
template <int E> __device__ __forceinline__ Piece<E> load_piece(const __nv_bfloat16* p) {
    Piece<E> r;
    if (E == 2) { const __nv_bfloat162 t = *reinterpret_cast<const __nv_bfloat162*>(p); r.v[0] = __low2float(t); r.v[E - 1] = __high2float(t); }
    else r.v[0] = __bfloat162float(p[0]);
    return r;
}
template <int E> __device__ __forceinline__ void store_piece(float* p, const Piece<E>& r) {
    if (E == 2) *reinterpret_cast<float2*>(p) = make_float2(r.v[0], r.v[E - 1]);
    else p[0] = r.v[0];
}
template <int E> __device__ __forceinline__ void store_piece(__nv_bfloat16* p, const Piece<E>& r) {
    if (E == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(r.v[0], r.v[E - 1]);
    else p[0] = __float2bfloat16_rn(r.v[0]);
}

// blockIdx.x is the token, blockIdx.y * 4 + warp the run of heads.
template <typename TI, typename TO, int E, int IT>
__global__ void __launch_bounds__(128) qk_norm_rope_pairs_kernel(const QkvParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int heads_total = p.nq + (p.kv_in_proj ? 2 * p.nkv : 0);
    const int t = blockIdx.x;
    const int head0 = (blockIdx.y * 4 + warp) * HEADS_PER_WARP;
    if (head0 >= heads_total || (head0 >= p.nq && !p.write_kv)) return;
    const int half = p.d >> 1;
    const TI* in = (const TI*)p.qkv + ((size_t)t * heads_total + head0) * p.d;

    // every load of the warp's heads is issued before the first store (the compiler cannot move loads across the
    // stores itself: it does not know that the projection and the outputs are different memory)
    Piece<E> lo[HEADS_PER_WARP][IT], hi[HEADS_PER_WARP][IT];
#pragma unroll
    for (int hh = 0; hh < HEADS_PER_WARP; ++hh) {
        const TI* src = in + (head0 + hh < heads_total ? hh : 0) * p.d;
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            const int j = (it * 32 + lane) * E;
            lo[hh][it] = load_piece<E>(src + j);
            hi[hh][it] = load_piece<E>(src + half + j);
        }
    }
    if (p.n_splits > 1) {
        for (int s = 1; s < p.n_splits; ++s) {
#pragma unroll
            for (int hh = 0; hh < HEADS_PER_WARP; ++hh) {
                const TI* src = in + (head0 + hh < heads_total ? hh : 0) * p.d + (size_t)s * p.split_stride;
#pragma unroll
                for (int it = 0; it < IT; ++it) {
                    const int j = (it * 32 + lane) * E;
                    const Piece<E> dl = load_piece<E>(src + j), dh = load_piece<E>(src + half + j);
#pragma unroll
                    for (int e = 0; e < E; ++e) { lo[hh][it].v[e] += dl.v[e]; hi[hh][it].v[e] += dh.v[e]; }
                }
            }
        }
    }
    // what all heads of the token share: position, cos and sin, the cache page, the norm weights
    const int pos = p.token_pos[t];
    const float* cs = p.cos_sin + (size_t)(pos < p.max_pos ? pos : p.max_pos - 1) * p.d;
    Piece<E> c[IT], sn[IT], wq_lo[IT], wq_hi[IT], wk_lo[IT], wk_hi[IT];
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int j = (it * 32 + lane) * E;
        c[it] = load_piece<E>(cs + j);
        sn[it] = load_piece<E>(cs + half + j);
        if (p.q_weight) { wq_lo[it] = load_piece<E>(p.q_weight + j); wq_hi[it] = load_piece<E>(p.q_weight + half + j); }
        if (p.k_weight) { wk_lo[it] = load_piece<E>(p.k_weight + j); wk_hi[it] = load_piece<E>(p.k_weight + half + j); }
    }
    size_t cache_row = 0;    // element offset of (page, kv head 0, token) in the caches
    if (p.write_kv && head0 + HEADS_PER_WARP > p.nq) {
        const int slot_pos = p.ring_tokens > 0 ? pos % p.ring_tokens : pos;
        const int page = p.block_table[(size_t)p.token_seq[t] * p.max_blocks + slot_pos / p.page_tokens];
        cache_row = ((size_t)page * p.nkv * p.page_tokens + (slot_pos % p.page_tokens)) * (size_t)p.d;
    }
    const size_t head_stride = (size_t)p.page_tokens * p.d;
    const float inv_d = 1.f / (float)p.d;
#pragma unroll
    for (int hh = 0; hh < HEADS_PER_WARP; ++hh) {
        const int head = head0 + hh;
        if (head >= heads_total) break;
        const bool is_q = head < p.nq, is_k = !is_q && head < p.nq + p.nkv;
        if (!is_q && !p.write_kv) break;
        TO* dst;
        if (is_q) dst = (TO*)p.q_out + ((size_t)t * p.nq + head) * p.d;
        else if (is_k) dst = (TO*)p.k_cache + cache_row + (size_t)(head - p.nq) * head_stride;
        else dst = (TO*)p.v_cache + cache_row + (size_t)(head - p.nq - p.nkv) * head_stride;
        const bool weighted = is_q ? p.q_weight != nullptr : (is_k && p.k_weight != nullptr);
        const bool normed = weighted || (p.unit_norm && (is_q || is_k));
        float inv = 1.f;
        if (normed) {
            float sq = 0.f;
#pragma unroll
            for (int it = 0; it < IT; ++it)
#pragma unroll
                for (int e = 0; e < E; ++e) sq += lo[hh][it].v[e] * lo[hh][it].v[e] + hi[hh][it].v[e] * hi[hh][it].v[e];
            inv = rsqrtf(warp_sum(sq) * inv_d + p.eps);
        }
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            const int j = (it * 32 + lane) * E;
            Piece<E> a = lo[hh][it], b = hi[hh][it];
            if (normed && !weighted) {
#pragma unroll
                for (int e = 0; e < E; ++e) { a.v[e] *= inv; b.v[e] *= inv; }
            } else if (normed) {
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    a.v[e] = a.v[e] * inv * (is_q ? wq_lo[it].v[e] : wk_lo[it].v[e]);
                    b.v[e] = b.v[e] * inv * (is_q ? wq_hi[it].v[e] : wk_hi[it].v[e]);
                }
            }
            if (is_q || is_k) {
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    const float ya = a.v[e] * c[it].v[e] - b.v[e] * sn[it].v[e];
                    const float yb = b.v[e] * c[it].v[e] + a.v[e] * sn[it].v[e];
                    a.v[e] = ya; b.v[e] = yb;
                }
            }
            store_piece<E>(dst + j, a);
            store_piece<E>(dst + half + j, b);
        }
    }
}

extern "C" int qt_qk_norm_rope_write(const void* qkv, int in_dtype, int n_splits, long long split_stride, void* q_out,
                                     void* k_cache, void* v_cache, int out_dtype, const int* token_seq,
                                     const int* token_pos, const int* block_table, int max_blocks,
                                     const float* q_weight, const float* k_weight, float eps, const float* cos_sin,
                                     int rotary_dim, int max_pos, int n_tokens, int nq, int nkv, int d, int page_tokens,
                                     int ring_tokens, int write_kv, int kv_in_proj, int interleaved, int nv, int dv, int unit_norm, int whole_norm,
                                     float* row_inv, int extra_cols, void* stream) {
    if (nv <= 0) nv = nkv;
    if (dv <= 0) dv = d;
    const bool own_values = nv != nkv || dv != d;
    QT_REQUIRE(extra_cols >= 0 && (!whole_norm || (row_inv && q_weight && (k_weight || !kv_in_proj) && !unit_norm)),
               "qk_norm_rope_write: a norm over the whole projection needs its factors' buffer and both weights");
    QT_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && d <= 1024, "qk_norm_rope_write: bad sizes T=%d nq=%d nkv=%d d=%d", n_tokens, nq, nkv, d);
    QT_REQUIRE(rotary_dim >= 0 && rotary_dim <= d && rotary_dim % 2 == 0, "qk_norm_rope_write: rotary_dim=%d must be even and at most head_dim=%d", rotary_dim, d);
    QT_REQUIRE(rotary_dim == 0 || (cos_sin && max_pos > 0), "qk_norm_rope_write: rotation needs a cos/sin table");
    QT_REQUIRE(page_tokens > 0 && n_splits >= 1 && ring_tokens >= 0, "qk_norm_rope_write: bad cache geometry");
    QT_REQUIRE(!write_kv || (k_cache && v_cache && block_table), "qk_norm_rope_write: cache pointers missing");
    QT_REQUIRE(!write_kv || kv_in_proj, "qk_norm_rope_write: nothing to write without k and v in the projection");
    if (n_tokens == 0) return QT_OK;
    QkvParams p{qkv, n_splits, (size_t)split_stride, q_out, k_cache, v_cache, token_seq, token_pos, block_table, max_blocks,
                q_weight, k_weight, eps, cos_sin, rotary_dim, max_pos, n_tokens, nq, nkv, d, page_tokens, ring_tokens, write_kv, kv_in_proj, interleaved, nv, dv,
                unit_norm, whole_norm ? row_inv : nullptr, extra_cols};
    const int warps = 4;
    const long long items = (long long)n_tokens * (nq + (kv_in_proj ? nkv + nv : 0));
    const unsigned grid = (unsigned)((items + warps - 1) / warps);
    const size_t smem = (size_t)warps * d * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    // 16-byte loads and stores need head_dim % 8 == 0 (bfloat16 rows of the cache and of q) and aligned bases
    // (q and k heads of a projection whose values have their own shape take them too, if the values' columns keep the rows aligned)
    if (whole_norm) {
        const size_t cols = (size_t)nq * d + (kv_in_proj ? (size_t)nkv * d + (size_t)nv * dv : 0) + (size_t)extra_cols;
        if (in_dtype == QT_F32)
            launch_kernel(qk_row_rms_kernel<float>, dim3(n_tokens), dim3(256), 0, s, (const float*)qkv, n_splits, (size_t)split_stride, cols, nq * d,
                          kv_in_proj ? nkv * d : 0, eps, row_inv);
        else if (in_dtype == QT_BF16)
            launch_kernel(qk_row_rms_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(256), 0, s, (const __nv_bfloat16*)qkv, n_splits, (size_t)split_stride, cols,
                          nq * d, kv_in_proj ? nkv * d : 0, eps, row_inv);
        else QT_FAIL(QT_ERR_ARG, "qk_norm_rope_write: unsupported element type %d", in_dtype);
        QT_CHECK_LAUNCH("qk_row_rms");
    }
    const bool vec = (!own_values || (nv * dv) % 8 == 0) && extra_cols % 8 == 0 && d % 8 == 0 && split_stride % 8 == 0 && ((uintptr_t)qkv % 16 == 0) && ((uintptr_t)q_out % 16 == 0) &&
                     (!write_kv || (((uintptr_t)k_cache % 16 == 0) && ((uintptr_t)v_cache % 16 == 0)));
    // the register form: all dimensions rotate, half a head is one or two rounds of 32 or 64 elements, enough tokens
    // to fill the machine with a few heads per warp
    const int half = d / 2;
    int pe = 0, pit = 0;
    if (interleaved) { pe = 0; }                     // the register form pairs (i, i + d/2)
    else if (rotary_dim == d && half % 64 == 0 && half / 64 <= 2) { pe = 2; pit = half / 64; }
    else if (rotary_dim == d && half == 32) { pe = 1; pit = 1; }
    const bool pair_aligned = split_stride % 2 == 0 && ((uintptr_t)qkv % 8 == 0) && ((uintptr_t)q_out % 8 == 0) && ((uintptr_t)cos_sin % 8 == 0) &&
                              (!q_weight || (uintptr_t)q_weight % 8 == 0) && (!k_weight || (uintptr_t)k_weight % 8 == 0) &&
                              (!write_kv || (((uintptr_t)k_cache % 8 == 0) && ((uintptr_t)v_cache % 8 == 0)));
    if (pe && !own_values && !(unit_norm && (q_weight || k_weight)) && !whole_norm && !extra_cols && pair_aligned && n_tokens >= 256 && nq + 2 * nkv <= 65535 * 16 && (in_dtype == QT_F32 || in_dtype == QT_BF16) && out_dtype == QT_BF16) {
        const int heads_total = nq + (kv_in_proj ? 2 * nkv : 0);
        const dim3 pgrid((unsigned)n_tokens, (unsigned)((heads_total + warps * HEADS_PER_WARP - 1) / (warps * HEADS_PER_WARP)));
#define QT_LAUNCH_PAIRS(TI, E, IT) launch_kernel(qk_norm_rope_pairs_kernel<TI, __nv_bfloat16, E, IT>, pgrid, dim3(warps * 32), 0, s, p)
        if (in_dtype == QT_BF16) {
            if (pe == 2 && pit == 1) QT_LAUNCH_PAIRS(__nv_bfloat16, 2, 1);
            else if (pe == 2) QT_LAUNCH_PAIRS(__nv_bfloat16, 2, 2);
            else QT_LAUNCH_PAIRS(__nv_bfloat16, 1, 1);
        } else {
            if (pe == 2 && pit == 1) QT_LAUNCH_PAIRS(float, 2, 1);
            else if (pe == 2) QT_LAUNCH_PAIRS(float, 2, 2);
            else QT_LAUNCH_PAIRS(float, 1, 1);
        }
#undef QT_LAUNCH_PAIRS
        QT_CHECK_LAUNCH("qk_norm_rope_write");
        return QT_OK;
    }
#define QT_LAUNCH_QKV(TI, TO)                                                                    \
    do {                                                                                         \
        if (vec) launch_kernel(qk_norm_rope_write_kernel<TI, TO, true>, dim3(grid), dim3(warps * 32), smem, s, p);      \
        else launch_kernel(qk_norm_rope_write_kernel<TI, TO, false>, dim3(grid), dim3(warps * 32), smem, s, p);         \
    } while (0)
    if (in_dtype == QT_F32 && out_dtype == QT_F32) QT_LAUNCH_QKV(float, float);
    else if (in_dtype == QT_F32 && out_dtype == QT_BF16) QT_LAUNCH_QKV(float, __nv_bfloat16);
    else if (in_dtype == QT_BF16 && out_dtype == QT_BF16) QT_LAUNCH_QKV(__nv_bfloat16, __nv_bfloat16);
    else QT_FAIL(QT_ERR_ARG, "qk_norm_rope_write: unsupported element types %d -> %d", in_dtype, out_dtype);
#undef QT_LAUNCH_QKV
    QT_CHECK_LAUNCH("qk_norm_rope_write");
    return QT_OK;
}

// ----------------------------------------------------------------------------- projection bias + value norm + value blend + cache write
// For mixers without rotation whose values are treated before they are cached.  Input: the fused projection output
// [t, nq * d + nkv * d + nkv * dv] (possibly split-K partial sums), the value head size dv free of the q/k size d.
// One warp per (token, head), everything in float:
//   q head:  + bias, store to q_out[t, h, :]
//   k head:  + bias, store into the key cache at the token's position
//   v head:  + bias; with v_norm divided by sqrt(mean(v^2) + v_eps); with blend_from,
//            v = (1 - lambda) v + lambda * blend_from[t, kv head, :], lambda read from the device;
//            with keep_to, keep_to[t, kv head, :] = v (float: what a later layer blends with);
//            store into the value cache.
struct QkvTreatParams {
    const void* qkv; int n_splits; size_t split_stride;
    const float* bias;                    // [nq * d + nkv * d + nkv * dv] or null
    void* q_out; void* k_cache; void* v_cache;
    const int* token_seq; const int* token_pos; const int* block_table; int max_blocks;
    int v_norm; float v_eps;
    const float* blend_from; const float* blend_lambda; float* keep_to;
    int n_tokens, nq, nkv, d, dv, page_tokens, ring_tokens, write_kv;
};

template <typename TI, typename TO>
__global__ void qkv_treat_write_kernel(const QkvTreatParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int heads_total = p.nq + 2 * p.nkv;
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= (long long)p.n_tokens * heads_total) return;
    const int t = (int)(item / heads_total);
    const int head = (int)(item % heads_total);
    const bool is_q = head < p.nq, is_k = !is_q && head < p.nq + p.nkv;
    if (!is_q && !p.write_kv) return;
    const int row_width = (p.nq + p.nkv) * p.d + p.nkv * p.dv;
    const int col0 = is_q ? head * p.d : (is_k ? p.nq * p.d + (head - p.nq) * p.d : (p.nq + p.nkv) * p.d + (head - p.nq - p.nkv) * p.dv);
    const int len = (is_q || is_k) ? p.d : p.dv;
    const TI* in = (const TI*)p.qkv + (size_t)t * row_width + col0;
    const float* bias = p.bias ? p.bias + col0 : nullptr;
    const int pos = p.token_pos[t];
    if (is_q || is_k) {
        TO* dst;
        if (is_q) dst = (TO*)p.q_out + ((size_t)t * p.nq + head) * p.d;
        else {
            const int* table = p.block_table + (size_t)p.token_seq[t] * p.max_blocks;
            dst = (TO*)p.k_cache + cache_offset(table, pos, p.ring_tokens, p.page_tokens, p.nkv, head - p.nq, p.d);
        }
        for (int i = lane; i < len; i += 32) {
            float x = load_sum(in, (size_t)i, p.n_splits, p.split_stride);
            if (bias) x += bias[i];
            dst[i] = from_float<TO>(x);
        }
        return;
    }
    const int kvh = head - p.nq - p.nkv;
    float sq = 0.f;
    for (int i = lane; i < len; i += 32) {
        float x = load_sum(in, (size_t)i, p.n_splits, p.split_stride);
        if (bias) x += bias[i];
        sq += x * x;
    }
    const float inv = p.v_norm ? 1.f / sqrtf(warp_sum(sq) / (float)len + p.v_eps) : 1.f;
    const float lambda = p.blend_from ? p.blend_lambda[0] : 0.f;
    const size_t side = ((size_t)t * p.nkv + kvh) * p.dv;
    const int* table = p.block_table + (size_t)p.token_seq[t] * p.max_blocks;
    TO* dst = (TO*)p.v_cache + cache_offset(table, pos, p.ring_tokens, p.page_tokens, p.nkv, kvh, p.dv);
    for (int i = lane; i < len; i += 32) {
        float x = load_sum(in, (size_t)i, p.n_splits, p.split_stride);       // read again: the row is in L1 or L2
        if (bias) x += bias[i];
        x *= inv;
        if (p.blend_from) x = (1.f - lambda) * x + lambda * p.blend_from[side + i];
        if (p.keep_to) p.keep_to[side + i] = x;
        dst[i] = from_float<TO>(x);
    }
}

// The same for head sizes that are multiples of 4 up to 256 and 16-byte aligned rows: a lane owns up to two pieces of
// four consecutive elements, sums the split-K partials with independent 16-byte loads and keeps the values in
// registers between the sum of squares and the stores.
template <typename TI, typename TO>
__global__ void qkv_treat_write_vec_kernel(const QkvTreatParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int heads_total = p.nq + 2 * p.nkv;
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= (long long)p.n_tokens * heads_total) return;
    const int t = (int)(item / heads_total);
    const int head = (int)(item % heads_total);
    const bool is_q = head < p.nq, is_k = !is_q && head < p.nq + p.nkv;
    if (!is_q && !p.write_kv) return;
    const int row_width = (p.nq + p.nkv) * p.d + p.nkv * p.dv;
    const int col0 = is_q ? head * p.d : (is_k ? p.nq * p.d + (head - p.nq) * p.d : (p.nq + p.nkv) * p.d + (head - p.nq - p.nkv) * p.dv);
    const int len = (is_q || is_k) ? p.d : p.dv;
    const int chunks = len >> 2;
    const TI* in = (const TI*)p.qkv + (size_t)t * row_width + col0;
    float4 x[2];
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int c = lane + 32 * i;
        if (c < chunks) {
            float4 v = load4(in + 4 * c);
            add_splits4<16>(v, in + 4 * c, 1, p.n_splits, p.split_stride);
            if (p.bias) { const float4 b = load4(p.bias + col0 + 4 * c); v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
            x[i] = v;
            sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    }
    const int pos = p.token_pos[t];
    TO* dst;
    if (is_q) dst = (TO*)p.q_out + ((size_t)t * p.nq + head) * p.d;
    else {
        const int* table = p.block_table + (size_t)p.token_seq[t] * p.max_blocks;
        dst = is_k ? (TO*)p.k_cache + cache_offset(table, pos, p.ring_tokens, p.page_tokens, p.nkv, head - p.nq, p.d)
                   : (TO*)p.v_cache + cache_offset(table, pos, p.ring_tokens, p.page_tokens, p.nkv, head - p.nq - p.nkv, p.dv);
    }
    if (is_q || is_k) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int c = lane + 32 * i;
            if (c < chunks) store4(dst + 4 * c, x[i]);
        }
        return;
    }
    const float inv = p.v_norm ? 1.f / sqrtf(warp_sum(sq) / (float)len + p.v_eps) : 1.f;
    const float lambda = p.blend_from ? p.blend_lambda[0] : 0.f;
    const size_t side = ((size_t)t * p.nkv + (head - p.nq - p.nkv)) * p.dv;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int c = lane + 32 * i;
        if (c < chunks) {
            float4 v = make_float4(x[i].x * inv, x[i].y * inv, x[i].z * inv, x[i].w * inv);
            if (p.blend_from) {
                const float4 o = load4(p.blend_from + side + 4 * c);
                v = make_float4((1.f - lambda) * v.x + lambda * o.x, (1.f - lambda) * v.y + lambda * o.y,
                                (1.f - lambda) * v.z + lambda * o.z, (1.f - lambda) * v.w + lambda * o.w);
            }
            if (p.keep_to) store4(p.keep_to + side + 4 * c, v);
            store4(dst + 4 * c, v);
        }
    }
}

extern "C" int qt_qkv_treat_write(const void* qkv, int in_dtype, int n_splits, long long split_stride, const float* bias,
                                  void* q_out, void* k_cache, void* v_cache, int out_dtype, const int* token_seq,
                                  const int* token_pos, const int* block_table, int max_blocks, int v_norm, float v_eps,
                                  const float* blend_from, const float* blend_lambda, float* keep_to, int n_tokens, int nq,
                                  int nkv, int d, int dv, int page_tokens, int ring_tokens, int write_kv, void* stream) {
    QT_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && dv > 0, "qkv_treat_write: bad sizes T=%d nq=%d nkv=%d d=%d dv=%d", n_tokens, nq, nkv, d, dv);
    QT_REQUIRE(page_tokens > 0 && n_splits >= 1 && ring_tokens >= 0, "qkv_treat_write: bad cache geometry");
    QT_REQUIRE(!write_kv || (k_cache && v_cache && block_table), "qkv_treat_write: cache pointers missing");
    QT_REQUIRE(!blend_from || blend_lambda, "qkv_treat_write: a blend needs its weight");
    QT_REQUIRE(!v_norm || v_eps > 0.f, "qkv_treat_write: the value norm needs a positive eps");
    if (n_tokens == 0) return QT_OK;
    QkvTreatParams p{qkv, n_splits, (size_t)split_stride, bias, q_out, k_cache, v_cache, token_seq, token_pos, block_table, max_blocks,
                     v_norm, v_eps, blend_from, blend_lambda, keep_to, n_tokens, nq, nkv, d, dv, page_tokens, ring_tokens, write_kv};
    const int warps = 4;
    const long long items = (long long)n_tokens * (nq + 2 * nkv);
    const unsigned grid = (unsigned)((items + warps - 1) / warps);
    cudaStream_t s = (cudaStream_t)stream;
    auto aligned = [](const void* ptr) { return ptr == nullptr || (uintptr_t)ptr % 16 == 0; };
    const bool vec = d % 4 == 0 && dv % 4 == 0 && d <= 256 && dv <= 256 && split_stride % 4 == 0 && aligned(qkv) && aligned(bias) && aligned(q_out) &&
                     aligned(k_cache) && aligned(v_cache) && aligned(blend_from) && aligned(keep_to);
    if (vec) {
        if (in_dtype == QT_F32 && out_dtype == QT_F32) launch_kernel(qkv_treat_write_vec_kernel<float, float>, dim3(grid), dim3(warps * 32), 0, s, p);
        else if (in_dtype == QT_F32 && out_dtype == QT_BF16) launch_kernel(qkv_treat_write_vec_kernel<float, __nv_bfloat16>, dim3(grid), dim3(warps * 32), 0, s, p);
        else if (in_dtype == QT_BF16 && out_dtype == QT_BF16) launch_kernel(qkv_treat_write_vec_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(grid), dim3(warps * 32), 0, s, p);
        else QT_FAIL(QT_ERR_ARG, "qkv_treat_write: unsupported element types %d -> %d", in_dtype, out_dtype);
        QT_CHECK_LAUNCH("qkv_treat_write");
        return QT_OK;
    }
    if (in_dtype == QT_F32 && out_dtype == QT_F32) launch_kernel(qkv_treat_write_kernel<float, float>, dim3(grid), dim3(warps * 32), 0, s, p);
    else if (in_dtype == QT_F32 && out_dtype == QT_BF16) launch_kernel(qkv_treat_write_kernel<float, __nv_bfloat16>, dim3(grid), dim3(warps * 32), 0, s, p);
    else if (in_dtype == QT_BF16 && out_dtype == QT_BF16) launch_kernel(qkv_treat_write_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(grid), dim3(warps * 32), 0, s, p);
    else QT_FAIL(QT_ERR_ARG, "qkv_treat_write: unsupported element types %d -> %d", in_dtype, out_dtype);
    QT_CHECK_LAUNCH("qkv_treat_write");
    return QT_OK;
}

// ----------------------------------------------------------------------------- gated product
// out[t, i] = act(g) * u (act: SiLU or another of QT_ACT_*); float inside.  Plain layout (group 0): g = gate_up[t, i], u = gate_up[t, inter + i].
// Interleaved layout (group G, the fused weight's rows alternate G of gate and G of up, which is what lets a GEMM
// epilogue see both in one warp): g = gate_up[t, (i / G) * 2G + i % G], u = the element G further on.  `bias` (or null)
// holds a float per column of gate_up, in its layout, added to the sums.
__device__ __forceinline__ size_t gate_column(int i, int group) { return group ? (size_t)(i / group) * 2 * group + i % group : (size_t)i; }

template <typename TI, typename TO>
__global__ void swiglu_kernel(const TI* __restrict__ gate_up, int n_splits, size_t split_stride, const float* __restrict__ bias,
                              TO* __restrict__ out, long long total, int inter, int group, int act, float limit) {
    pdl_launch_dependents();
    pdl_wait();
    const int up_offset = group ? group : inter;
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (long long)gridDim.x * blockDim.x) {
        const long long t = idx / inter;
        const int i = (int)(idx % inter);
        const size_t base = (size_t)t * 2 * inter + gate_column(i, group);
        float g = load_sum(gate_up, base, n_splits, split_stride);
        float u = load_sum(gate_up, base + up_offset, n_splits, split_stride);
        if (bias) { const int at = (int)gate_column(i, group); g += bias[at]; u += bias[at + up_offset]; }
        out[idx] = from_float<TO>(gated_value<false>(g, u, act, limit));
    }
}

// Eight elements per thread with 16- or 32-byte loads and stores (widths that are multiples of 8, aligned bases).
// blockIdx.x is the token, blockIdx.y a run of chunks of its row.
struct Float8 { float4 a, b; };
__device__ __forceinline__ Float8 load8(const float* p) { return {load4(p), load4(p + 4)}; }
__device__ __forceinline__ Float8 load8(const __nv_bfloat16* p) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    return {make_float4(__low2float(h[0]), __high2float(h[0]), __low2float(h[1]), __high2float(h[1])),
            make_float4(__low2float(h[2]), __high2float(h[2]), __low2float(h[3]), __high2float(h[3]))};
}
__device__ __forceinline__ void store8(float* p, const Float8& v) { store4(p, v.a); store4(p + 4, v.b); }
__device__ __forceinline__ void store8(__nv_bfloat16* p, const Float8& v) {
    __nv_bfloat162 h[4] = {__floats2bfloat162_rn(v.a.x, v.a.y), __floats2bfloat162_rn(v.a.z, v.a.w),
                           __floats2bfloat162_rn(v.b.x, v.b.y), __floats2bfloat162_rn(v.b.z, v.b.w)};
    *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(h);
}
__device__ __forceinline__ void add4(float4& x, const float4& y) { x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w; }
// silu(g) * u.  For a float result the exponential and the division are the library's; for a bfloat16 result
// (8 bits of mantissa) the hardware approximations (2 ulp of float) are used: with the exact forms the kernel was
// bound by instruction issue, not by memory.
template <typename TO> __device__ __forceinline__ float silu_mul(float g, float u, int act, float limit) { return gated_value<false>(g, u, act, limit); }
template <> __device__ __forceinline__ float silu_mul<__nv_bfloat16>(float g, float u, int act, float limit) { return gated_value<true>(g, u, act, limit); }
template <typename TO> __device__ __forceinline__ float4 silu_mul4(const float4& g, const float4& u, int act, float limit) {
    return make_float4(silu_mul<TO>(g.x, u.x, act, limit), silu_mul<TO>(g.y, u.y, act, limit), silu_mul<TO>(g.z, u.z, act, limit),
                       silu_mul<TO>(g.w, u.w, act, limit));
}

// PT chunks per thread, all loads issued before the first store.
template <typename TI, typename TO, int PT>
__global__ void swiglu_vec_kernel(const TI* __restrict__ gate_up, int n_splits, size_t split_stride, const float* __restrict__ bias,
                                  TO* __restrict__ out, int inter, int group, int act, float limit) {
    pdl_launch_dependents();
    pdl_wait();
    const int chunks = inter >> 3;
    const int up_offset = group ? group : inter;
    const TI* row = gate_up + (size_t)blockIdx.x * 2 * inter;
    TO* orow = out + (size_t)blockIdx.x * inter;
    for (int c0 = blockIdx.y * blockDim.x * PT + threadIdx.x; c0 < chunks; c0 += gridDim.y * blockDim.x * PT) {
        Float8 g[PT], u[PT];
#pragma unroll
        for (int i = 0; i < PT; ++i) {
            const int c = c0 + i * blockDim.x;
            if (c < chunks) { const size_t at = gate_column(8 * c, group); g[i] = load8(row + at); u[i] = load8(row + at + up_offset); }
        }
        for (int s = 1; s < n_splits; ++s) {
#pragma unroll
            for (int i = 0; i < PT; ++i) {
                const int c = c0 + i * blockDim.x;
                if (c < chunks) {
                    const size_t at = gate_column(8 * c, group) + (size_t)s * split_stride;
                    const Float8 dg = load8(row + at), du = load8(row + at + up_offset);
                    add4(g[i].a, dg.a); add4(g[i].b, dg.b); add4(u[i].a, du.a); add4(u[i].b, du.b);
                }
            }
        }
        if (bias) {
#pragma unroll
            for (int i = 0; i < PT; ++i) {
                const int c = c0 + i * blockDim.x;
                if (c < chunks) {
                    const size_t at = gate_column(8 * c, group);
                    const Float8 bg = load8(bias + at), bu = load8(bias + at + up_offset);
                    add4(g[i].a, bg.a); add4(g[i].b, bg.b); add4(u[i].a, bu.a); add4(u[i].b, bu.b);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < PT; ++i) {
            const int c = c0 + i * blockDim.x;
            if (c < chunks) store8(orow + 8 * c, Float8{silu_mul4<TO>(g[i].a, u[i].a, act, limit), silu_mul4<TO>(g[i].b, u[i].b, act, limit)});
        }
    }
}

extern "C" int qt_swiglu(const void* gate_up, int in_dtype, int n_splits, long long split_stride, const float* bias, void* out, int out_dtype,
                         int n_tokens, int inter, int group, int act, float limit, void* stream) {
    QT_REQUIRE(act >= 0 && act <= QT_ACT_CAPPED, "swiglu: unknown activation code %d", act);
    QT_REQUIRE(n_tokens >= 0 && inter > 0 && n_splits >= 1, "swiglu: bad sizes T=%d I=%d", n_tokens, inter);
    QT_REQUIRE(group >= 0 && (group == 0 || inter % group == 0), "swiglu: rows interleaved in groups of %d do not divide I=%d", group, inter);
    if (n_tokens == 0) return QT_OK;
    const long long total = (long long)n_tokens * inter;
    const int threads = 256;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = inter % 8 == 0 && group % 8 == 0 && split_stride % 8 == 0 && ((uintptr_t)gate_up % 16 == 0) && ((uintptr_t)out % 16 == 0) &&
                     ((uintptr_t)bias % 16 == 0);
    long long blocks = (total + threads - 1) / threads;
    if (blocks > (long long)sm_count() * 16) blocks = (long long)sm_count() * 16;
    // few tokens (decode): one chunk per thread, most blocks; many tokens (prefill): two chunks per thread
    const int per_thread = n_tokens >= 256 ? 2 : 1;
    unsigned per_row = (unsigned)((inter / 8 + threads * per_thread - 1) / (threads * per_thread));
    if (per_row > 65535u) per_row = 65535u;
#define QT_LAUNCH_SWIGLU(TI, TO)                                                                                              \
    do {                                                                                                                      \
        if (vec && per_thread == 2) launch_kernel(swiglu_vec_kernel<TI, TO, 2>, dim3((unsigned)n_tokens, per_row), dim3(threads), 0, s, \
                               (const TI*)gate_up, n_splits, (size_t)split_stride, bias, (TO*)out, inter, group, act, limit);              \
        else if (vec) launch_kernel(swiglu_vec_kernel<TI, TO, 1>, dim3((unsigned)n_tokens, per_row), dim3(threads), 0, s,     \
                               (const TI*)gate_up, n_splits, (size_t)split_stride, bias, (TO*)out, inter, group, act, limit);              \
        else launch_kernel(swiglu_kernel<TI, TO>, dim3((unsigned)blocks), dim3(threads), 0, s, (const TI*)gate_up, n_splits,  \
                           (size_t)split_stride, bias, (TO*)out, total, inter, group, act, limit);                                         \
    } while (0)
    if (in_dtype == QT_F32 && out_dtype == QT_F32) QT_LAUNCH_SWIGLU(float, float);
    else if (in_dtype == QT_F32 && out_dtype == QT_BF16) QT_LAUNCH_SWIGLU(float, __nv_bfloat16);
    else if (in_dtype == QT_BF16 && out_dtype == QT_BF16) QT_LAUNCH_SWIGLU(__nv_bfloat16, __nv_bfloat16);
    else QT_FAIL(QT_ERR_ARG, "swiglu: unsupported element types %d -> %d", in_dtype, out_dtype);
#undef QT_LAUNCH_SWIGLU
    QT_CHECK_LAUNCH("swiglu");
    return QT_OK;
}

QT_DEFINE_LAST_ERROR(elementwise)
