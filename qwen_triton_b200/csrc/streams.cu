// A residual of several parallel streams ("hyper-connections"): S copies x_1 .. x_S of a token's row, kept as [T, S, H] floats.
// A sublayer reads u = sum_s read[s] x_s through its norm; its result y comes back as
//     x_t <- sum_s mix[s][t] x_s + out[t] y          (all t at once, from the old streams; `out` carries the constant factor)
// What is between two sublayers is one pass over the streams: the update by the sublayer before, the read of the one behind and
// its RMS norm.
//
// streams_norm_vec_kernel      one block per row, four elements of every stream per thread and round
// streams_norm_cluster_kernel  few rows: a cluster of blocks per row, which exchange their shares of the sum of squares
// streams_norm_kernel          any width and stream count
#include "common.cuh"

using namespace qt;

namespace {

constexpr int MAX_STREAMS = 32;    // of the general kernel
constexpr int VEC_STREAMS = 8;     // of the two vector kernels
constexpr int CACHE = 4;           // rounds of four elements that a thread keeps between the two passes
constexpr int CLUSTER = 8;

struct StreamArgs {
    float* streams;                                            // [T, S, H]
    const float* delta; int n_splits; size_t split_stride;     // y [splits, T, H], or null: the streams stay as they are
    const float* mix; const float* out_weight;                 // [S][S] (from, to) and [S]
    const float* read;                                         // [S], or null: ones
    const float* weight; float eps;                            // [H]
    const int* rows;                                           // or null: every row, and the streams are updated in place
    int hidden, streams_count;
};

__device__ __forceinline__ float4 get4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, const float4& v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&a);
    raw.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ void add_scaled(float4& d, float f, const float4& v) {
    d.x = fmaf(f, v.x, d.x); d.y = fmaf(f, v.y, d.y); d.z = fmaf(f, v.z, d.z); d.w = fmaf(f, v.w, d.w);
}
__device__ __forceinline__ float square4(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// The sublayer's result at four neighbouring elements: the planes of a split product added in their order, BATCH loads in flight.
template <int BATCH>
__device__ __forceinline__ float4 sum_planes4(const float* p, int n_splits, size_t stride) {
    float4 y = get4(p);
    for (int s0 = 1; s0 < n_splits; s0 += BATCH) {
        float4 t[BATCH];
#pragma unroll
        for (int j = 0; j < BATCH; ++j) t[j] = get4(p + (size_t)min(s0 + j, n_splits - 1) * stride);
#pragma unroll
        for (int j = 0; j < BATCH; ++j)
            if (s0 + j < n_splits) { y.x += t[j].x; y.y += t[j].y; y.z += t[j].z; y.w += t[j].w; }
    }
    return y;
}

// The weights of the update and of the read, the same for every token: they belong to the model, not to a kernel before this
// one, so they are fetched ahead of the wait.
template <int S> struct Weights {
    float mix[S * S], out[S], read[S];
    __device__ __forceinline__ Weights(const StreamArgs& p) {
#pragma unroll
        for (int t = 0; t < S; ++t) {
            read[t] = p.read ? __ldg(p.read + t) : 1.f;
            out[t] = p.delta ? __ldg(p.out_weight + t) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < S * S; ++i) mix[i] = p.delta ? __ldg(p.mix + i) : 0.f;
    }
};

// Four elements of a row: updates the streams (and stores them where `store`), returns what the next sublayer reads.
template <int S, int BATCH>
__device__ __forceinline__ float4 step4(const StreamArgs& p, const Weights<S>& w, size_t row, int c, bool store) {
    float* at = p.streams + row * S * p.hidden + 4 * c;
    float4 x[S];
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = get4(at + (size_t)s * p.hidden);
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!p.delta) {
#pragma unroll
        for (int s = 0; s < S; ++s) add_scaled(u, w.read[s], x[s]);
        return u;
    }
    const float4 y = sum_planes4<BATCH>(p.delta + row * p.hidden + 4 * c, p.n_splits, p.split_stride);
#pragma unroll
    for (int t = 0; t < S; ++t) {
        float4 v = make_float4(w.out[t] * y.x, w.out[t] * y.y, w.out[t] * y.z, w.out[t] * y.w);
#pragma unroll
        for (int s = 0; s < S; ++s) add_scaled(v, w.mix[s * S + t], x[s]);
        if (store) put4(at + (size_t)t * p.hidden, v);
        add_scaled(u, w.read[t], v);
    }
    return u;
}

template <int S, typename TO>
__global__ void __launch_bounds__(1024) streams_norm_vec_kernel(const StreamArgs p, TO* __restrict__ out) {
    pdl_launch_dependents();
    __shared__ float scratch[32];
    const Weights<S> w(p);
    pdl_wait();
    const int r = blockIdx.x;
    const size_t src = p.rows ? p.rows[r] : r;
    const int chunks = p.hidden >> 2;
    float4 u[CACHE];
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < CACHE; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
            u[i] = step4<S, 4>(p, w, src, c, !p.rows);
            sq += square4(u[i]);
        }
    }
    const float inv = rsqrtf(block_sum(sq, scratch) / (float)p.hidden + p.eps);
#pragma unroll
    for (int i = 0; i < CACHE; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
            const float4 g = get4(p.weight + 4 * c);
            put4(out + (size_t)r * p.hidden + 4 * c, make_float4(u[i].x * inv * g.x, u[i].y * inv * g.y, u[i].z * inv * g.z, u[i].w * inv * g.w));
        }
    }
}

// One chunk of four elements per thread; the blocks' shares of the sum of squares go to every block of the cluster.
template <int S, typename TO>
__global__ void __launch_bounds__(1024) streams_norm_cluster_kernel(const StreamArgs p, TO* __restrict__ out) {
    pdl_launch_dependents();
    cluster_arrive_started();
    __shared__ float scratch[32];
    __shared__ float shares[CLUSTER];
    const Weights<S> w(p);
    const uint32_t rank = cluster_rank();
    const int r = blockIdx.x / CLUSTER, chunks = p.hidden >> 2;
    const int c = (int)rank * blockDim.x + threadIdx.x;
    const float4 g = c < chunks ? get4(p.weight + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
    pdl_wait();
    const size_t src = p.rows ? p.rows[r] : r;
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < chunks) u = step4<S, 15>(p, w, src, c, !p.rows);
    const float share = block_sum(square4(u), scratch);
    cluster_wait_started();
    if (threadIdx.x < CLUSTER) cluster_store_float(&shares[rank], threadIdx.x, share);
    cluster_barrier();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < CLUSTER; ++i) total += shares[i];
    const float inv = rsqrtf(total / (float)p.hidden + p.eps);
    if (c < chunks) put4(out + (size_t)r * p.hidden + 4 * c, make_float4(u.x * inv * g.x, u.y * inv * g.y, u.z * inv * g.z, u.w * inv * g.w));
}

// One block per row, one element of every stream per thread and round.
template <typename TO>
__global__ void streams_norm_kernel(const StreamArgs p, TO* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int r = blockIdx.x, S = p.streams_count;
    const size_t src = p.rows ? p.rows[r] : r;
    float* row = p.streams + src * S * p.hidden;
    auto read = [&](int s) { return p.read ? __ldg(p.read + s) : 1.f; };
    auto value = [&](int i, bool update, bool store) {          // what the next sublayer reads at element i
        float x[MAX_STREAMS], u = 0.f;
        for (int s = 0; s < S; ++s) x[s] = row[(size_t)s * p.hidden + i];
        if (!update) {
            for (int s = 0; s < S; ++s) u = fmaf(read(s), x[s], u);
            return u;
        }
        const float y = load_sum(p.delta, src * p.hidden + i, p.n_splits, p.split_stride);
        for (int t = 0; t < S; ++t) {
            float v = __ldg(p.out_weight + t) * y;
            for (int s = 0; s < S; ++s) v = fmaf(__ldg(p.mix + s * S + t), x[s], v);
            if (store) row[(size_t)t * p.hidden + i] = v;
            u = fmaf(read(t), v, u);
        }
        return u;
    };
    float sq = 0.f;
    for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
        const float u = value(i, p.delta != nullptr, !p.rows);
        sq += u * u;
    }
    const float inv = rsqrtf(block_sum(sq, scratch) / (float)p.hidden + p.eps);
    // a thread reads again what it wrote itself; rows that are only listed are formed again
    for (int i = threadIdx.x; i < p.hidden; i += blockDim.x)
        out[(size_t)r * p.hidden + i] = from_float<TO>(value(i, p.delta != nullptr && p.rows, false) * inv * __ldg(p.weight + i));
}

template <int S, typename TO>
void launch_vec(const StreamArgs& p, TO* out, int n_rows, bool cluster, cudaStream_t s) {
    if (cluster) {
        const int per_block = (p.hidden / 4 + CLUSTER - 1) / CLUSTER;
        launch_kernel_cluster(streams_norm_cluster_kernel<S, TO>, dim3(n_rows * CLUSTER), dim3((per_block + 31) / 32 * 32), 0, s, CLUSTER, p, out);
    } else {
        const int per_thread = (p.hidden / 4 + CACHE - 1) / CACHE;
        int threads = (per_thread + 31) / 32 * 32;
        if (threads < 128) threads = 128;
        launch_kernel(streams_norm_vec_kernel<S, TO>, dim3(n_rows), dim3(threads), 0, s, p, out);
    }
}

template <typename TO>
int run(const StreamArgs& p, TO* out, int n_rows, cudaStream_t s) {
    const bool aligned = p.hidden % 4 == 0 && (uintptr_t)p.streams % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)p.weight % 16 == 0 &&
                         (!p.delta || ((uintptr_t)p.delta % 16 == 0 && p.split_stride % 4 == 0));
    const bool cluster = n_rows < 256 && p.hidden >= 4 * 32 * CLUSTER && p.hidden <= 4 * 1024 * CLUSTER;
    if (aligned && p.streams_count <= VEC_STREAMS && p.hidden <= 4 * 1024 * CACHE) {
        switch (p.streams_count) {
            case 1: launch_vec<1>(p, out, n_rows, cluster, s); break;
            case 2: launch_vec<2>(p, out, n_rows, cluster, s); break;
            case 3: launch_vec<3>(p, out, n_rows, cluster, s); break;
            case 4: launch_vec<4>(p, out, n_rows, cluster, s); break;
            case 5: launch_vec<5>(p, out, n_rows, cluster, s); break;
            case 6: launch_vec<6>(p, out, n_rows, cluster, s); break;
            case 7: launch_vec<7>(p, out, n_rows, cluster, s); break;
            default: launch_vec<8>(p, out, n_rows, cluster, s); break;
        }
    } else {
        launch_kernel(streams_norm_kernel<TO>, dim3(n_rows), dim3(256), 0, s, p, out);
    }
    QT_CHECK_LAUNCH("streams_norm");
    return QT_OK;
}

}  // namespace

extern "C" int qt_streams_norm(float* streams, const float* delta, int n_splits, long long split_stride, const float* mix, const float* out_weight,
                               const float* read, const float* weight, float eps, void* out, int out_dtype, const int* rows, int n_rows, int hidden,
                               int streams_count, void* stream) {
    QT_REQUIRE(n_rows >= 0 && hidden > 0 && n_splits >= 1 && streams_count >= 1 && streams_count <= MAX_STREAMS, "streams_norm: bad sizes rows=%d H=%d streams=%d (1..%d)",
               n_rows, hidden, streams_count, MAX_STREAMS);
    QT_REQUIRE(eps > 0.f && weight && out, "streams_norm: a norm needs a positive eps and a weight");
    QT_REQUIRE(!delta || (mix && out_weight), "streams_norm: an addition needs the weights it is written with");
    if (n_rows == 0) return QT_OK;
    const StreamArgs p{streams, delta, n_splits, (size_t)split_stride, mix, out_weight, read, weight, eps, rows, hidden, streams_count};
    return QT_DISPATCH_DTYPE(out_dtype, "streams_norm", { return run<T>(p, (T*)out, n_rows, (cudaStream_t)stream); });
}

QT_DEFINE_LAST_ERROR(streams)
