// The recurrence S <- diag(e^{g_t}) S + k_t v_t^T, o_t = S^T q_t with decays that depend on the token, for long steps: the
// tokens of a sequence are cut into chunks of CT = 64, everything a chunk does by itself runs for all chunks of all
// heads at once, and only the states pass from chunk to chunk.  With S_c the state in front of a chunk and G(s, t) the sum of
// the decays' logarithms g of the tokens s + 1 .. t,
//     o_t     = S_c^T (e^{G(start, t)} q_t) + sum_{s <= t} A[t, s] v_s,      A[t, s] = sum_n q_t[n] k_s[n] e^{G(s, t)[n]}
//     S_{c+1} = diag(e^{G(start, end)}) S_c + sum_s (e^{G(s, end)} k_s) v_s^T
// Every exponent is a sum of logarithms of decays over a range of tokens, so it is <= 0, nothing is divided by a decay and no
// two large sums are subtracted (per channel: running sums inside runs of 16 tokens, in the direction they are needed,
// and products of whole runs between them; per head: running sums in double).  All float; results differ from the
// token-by-token kernels by rounding only.
//
// chunk_prepare_channel_kernel   g per key channel: A (transposed, [s][t]), e^{G(start, t)} q_t, e^{G(s, end)} k_s and
//                                e^{G(start, end)} of a (chunk, head).
// chunk_prepare_head_kernel      g per head: A = (q_t . k_s) e^{G(s, t)} times the factor on v_s, and per token e^{G(start, t)} and
//                                e^{G(s, end)} times that factor; q and k themselves (which several heads may share) stay as they are.
// chunk_write_kernel             sum_s (e^{G(s, end)} k_s) v_s^T of a (chunk, head): a 64 x 64 x 64 product per tile.
// chunk_pass_kernel              walks a sequence's chunks elementwise: puts S_c in the place of what chunk c writes, and the last
//                                state back into the sequence's row.
// chunk_read_kernel              o of a (chunk, head): two products per 64 x 64 tile, over the state's rows and over the chunk's tokens.
//
// The chunk c of sequence i has the scratch index seq_start[i] / CT + i + c, which is below T / CT + (sequences) and distinct
// for distinct chunks.  States (and their scratch) are stored transposed, [heads, vdim, dim], as in linear_attention.cu.
#include "common.cuh"

#include <math.h>

using namespace qt;

namespace {

constexpr int CT = 64;             // tokens per chunk
constexpr int SUB = 16;            // tokens per run inside a chunk
constexpr int RUNS = CT / SUB;

struct ChunkArgs {
    const float* rows; int cols;                    // [T, cols]: q, k and v are columns of a token's row
    int at_q, at_k, at_v;
    const float* log_decay;                         // [T, heads, dim] or [T, heads]
    const float* v_scale;                           // [T, heads] or null
    float out_scale;                                // factor on q
    float* state;                                   // [slots + 1, heads, vdim, dim]
    float* out;                                     // [T, heads, vdim]
    const int* seq_start; const int* slots;
    int heads, heads_per_key, dim, vdim;
    float* states;                                  // [chunks, heads, vdim, dim]
    float* within;                                  // [chunks, heads, CT (s), CT (t)]
    float* whole;                                   // [chunks, heads, dim] or [chunks, heads]: e^{G(start, end)}
    float* q_from;                                  // per channel [T, heads, dim]: e^{G(start, t)} q_t; per head [T, heads]: the factor alone
    float* k_to;                                    // the same for e^{G(s, end)} k_s (per head: times v_scale)
};

struct Chunk { int first, count, index; };          // first token (of the step), tokens, scratch index; count <= 0: no such chunk

__device__ __forceinline__ Chunk chunk_of(const ChunkArgs& p, int seq, int c) {
    const int begin = p.seq_start[seq], end = p.seq_start[seq + 1];
    return {begin + c * CT, min(CT, end - begin - c * CT), begin / CT + seq + c};
}

// ----------------------------------------------------------------------------- decays per key channel
// grid (chunks of the longest sequence, heads, sequences), 256 threads; dynamic shared memory 3 CT (dim + 4) + CT (CT + 1) + 7 dim floats.
__global__ void __launch_bounds__(256) chunk_prepare_channel_kernel(const ChunkArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const int dim = p.dim, ld = dim + 4, head = blockIdx.y, key_head = head / p.heads_per_key;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x);
    if (ck.count <= 0) return;
    float* qs = sm;                        // [CT][ld] q, later e^{sum of its run up to t} q
    float* ks = qs + CT * ld;              // [CT][ld] k, later e^{sum of its run behind s} k
    float* as = ks + CT * ld;              // [CT][ld] e^{g}
    float* tile = as + CT * ld;            // [CT][CT + 1] A, row t
    float* run = tile + CT * (CT + 1);     // [RUNS][dim] sum of g over a run
    float* over = run + RUNS * dim;        // [3][dim] e^{run 1}, e^{run 2}, e^{run 1 + run 2}
    const float* g = p.log_decay + ((size_t)ck.first * p.heads + head) * dim;
    const size_t g_row = (size_t)p.heads * dim;
    for (int i = threadIdx.x; i < CT * dim; i += 256) {
        const int t = i / dim, n = i % dim;
        const bool in = t < ck.count;
        const size_t row = (size_t)(ck.first + t) * p.cols + (size_t)key_head * dim + n;
        qs[t * ld + n] = in ? p.rows[row + p.at_q] * p.out_scale : 0.f;
        ks[t * ld + n] = in ? p.rows[row + p.at_k] : 0.f;
        as[t * ld + n] = in ? expf(g[t * g_row + n]) : 1.f;
    }
    for (int i = threadIdx.x; i < CT * (CT + 1); i += 256) tile[i] = 0.f;
    __syncthreads();
    // inside a run: one warp per s; its lanes hold k_s decayed so far, multiplied by e^{g_t} as t goes on
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int s = warp; s < ck.count; s += 8) {
        const int r0 = s / SUB * SUB;
        float part[SUB];
#pragma unroll
        for (int j = 0; j < SUB; ++j) part[j] = 0.f;
        for (int n = lane; n < dim; n += 32) {
            float w = ks[s * ld + n];
#pragma unroll
            for (int j = 0; j < SUB; ++j) {
                const int t = r0 + j;
                if (t > s) w *= as[t * ld + n];
                if (t >= s) part[j] += w * qs[t * ld + n];
            }
        }
        // sixteen sums over the lanes: halve the values a lane carries four times, then one more exchange
#pragma unroll
        for (int half = SUB / 2; half >= 1; half >>= 1) {
            const bool upper = (lane & half) != 0;
#pragma unroll
            for (int j = 0; j < half; ++j) {
                const float give = upper ? part[j] : part[j + half], keep = upper ? part[j + half] : part[j];
                part[j] = keep + __shfl_xor_sync(0xffffffffu, give, half);
            }
        }
        const float total = part[0] + __shfl_xor_sync(0xffffffffu, part[0], 16);
        if (lane < SUB && r0 + lane >= s) tile[(r0 + lane) * (CT + 1) + s] = total;
    }
    __syncthreads();
    // running sums inside the runs, forwards on q and backwards on k
    for (int i = threadIdx.x; i < RUNS * dim; i += 256) {
        const int r = i / dim, n = i % dim;
        float v[SUB];
#pragma unroll
        for (int j = 0; j < SUB; ++j) v[j] = r * SUB + j < ck.count ? g[(size_t)(r * SUB + j) * g_row + n] : 0.f;
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < SUB; ++j) { sum += v[j]; qs[(r * SUB + j) * ld + n] *= expf(sum); }
        run[i] = sum;
        float behind = 0.f;
#pragma unroll
        for (int j = SUB - 1; j >= 0; --j) { ks[(r * SUB + j) * ld + n] *= expf(behind); behind += v[j]; }
    }
    __syncthreads();
    for (int n = threadIdx.x; n < dim; n += 256) {
        over[n] = expf(run[dim + n]);
        over[dim + n] = expf(run[2 * dim + n]);
        over[2 * dim + n] = expf(run[dim + n] + run[2 * dim + n]);
        p.whole[((size_t)ck.index * p.heads + head) * dim + n] = expf(run[n] + run[dim + n] + run[2 * dim + n] + run[3 * dim + n]);
    }
    __syncthreads();
    // between runs: A of run i against run j < i, two t by two s per thread
    for (int item = threadIdx.x; item < 6 * 64; item += 256) {
        const int pair = item >> 6, local = item & 63;
        const int i = pair < 1 ? 1 : pair < 3 ? 2 : 3, j = pair < 1 ? 0 : pair < 3 ? pair - 1 : pair - 3;
        const int t = i * SUB + (local >> 3) * 2, s = j * SUB + (local & 7) * 2;
        const float* mid = i - j == 3 ? over + 2 * dim : i - j == 2 ? (j == 0 ? over : over + dim) : nullptr;
        if (t >= ck.count) continue;
        float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
        const float *q0 = qs + t * ld, *q1 = q0 + ld, *k0 = ks + s * ld, *k1 = k0 + ld;
        for (int n = 0; n < dim; ++n) {
            float x0 = k0[n], x1 = k1[n];
            if (mid) { x0 *= mid[n]; x1 *= mid[n]; }
            a00 += q0[n] * x0; a01 += q0[n] * x1; a10 += q1[n] * x0; a11 += q1[n] * x1;
        }
        tile[t * (CT + 1) + s] = a00; tile[t * (CT + 1) + s + 1] = a01;
        tile[(t + 1) * (CT + 1) + s] = a10; tile[(t + 1) * (CT + 1) + s + 1] = a11;
    }
    // the decayed q and k of the whole chunk
    for (int i = threadIdx.x; i < ck.count * dim; i += 256) {
        const int t = i / dim, n = i % dim, r = t / SUB;
        float before = 0.f, after = 0.f;
#pragma unroll
        for (int o = 0; o < RUNS; ++o) { if (o < r) before += run[o * dim + n]; if (o > r) after += run[o * dim + n]; }
        const size_t at = ((size_t)(ck.first + t) * p.heads + head) * dim + n;
        p.q_from[at] = qs[t * ld + n] * expf(before);
        p.k_to[at] = ks[t * ld + n] * expf(after);
    }
    __syncthreads();
    float* within = p.within + ((size_t)ck.index * p.heads + head) * CT * CT;
    for (int i = threadIdx.x; i < CT * CT; i += 256) within[i] = tile[(i % CT) * (CT + 1) + i / CT];
}

// ----------------------------------------------------------------------------- tiles of products
constexpr int TILE = 64, KS = 16, LD = TILE + 4;

// acc[8][4] += X^T Y for X [KS][TILE], Y [KS][TILE] in shared memory (rows LD apart): thread ty owns rows 8 ty .., tx columns 4 tx ..
__device__ __forceinline__ void tile_fma(const float* xs, const float* ys, float (&acc)[8][4], int ty, int tx) {
#pragma unroll
    for (int k = 0; k < KS; ++k) {
        const float4 a0 = *reinterpret_cast<const float4*>(xs + k * LD + 8 * ty), a1 = *reinterpret_cast<const float4*>(xs + k * LD + 8 * ty + 4);
        const float4 b = *reinterpret_cast<const float4*>(ys + k * LD + 4 * tx);
        const float a[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            acc[i][0] = fmaf(a[i], b.x, acc[i][0]); acc[i][1] = fmaf(a[i], b.y, acc[i][1]);
            acc[i][2] = fmaf(a[i], b.z, acc[i][2]); acc[i][3] = fmaf(a[i], b.w, acc[i][3]);
        }
    }
}

constexpr int PT_THREADS = 128, PT_LOADS = TILE * KS / PT_THREADS;      // elements of a slice per thread

// One slice of KS rows of a 64 x 64 product: x(k, i) and y(k, i) give elements (0 outside), with i or k running fastest over
// neighbouring threads as the operand lies in memory.  The slice after next is fetched into registers under the arithmetic.
template <bool X_K_FAST, bool Y_K_FAST, typename FX, typename FY>
__device__ __forceinline__ void tile_product(int depth, FX x, FY y, float (&acc)[8][4], float* xs, float* ys) {
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float xr[PT_LOADS], yr[PT_LOADS];
    auto place = [&](int j, bool k_fast, int& k, int& i) {
        const int e = threadIdx.x + j * PT_THREADS;
        if (k_fast) { k = e % KS; i = e / KS; } else { k = e / TILE; i = e % TILE; }
    };
    auto fetch = [&](int k0) {
#pragma unroll
        for (int j = 0; j < PT_LOADS; ++j) {
            int k, i;
            place(j, X_K_FAST, k, i);
            xr[j] = k0 + k < depth ? x(k0 + k, i) : 0.f;
            place(j, Y_K_FAST, k, i);
            yr[j] = k0 + k < depth ? y(k0 + k, i) : 0.f;
        }
    };
    fetch(0);
    for (int k0 = 0; k0 < depth; k0 += KS) {
        __syncthreads();
#pragma unroll
        for (int j = 0; j < PT_LOADS; ++j) {
            int k, i;
            place(j, X_K_FAST, k, i);
            xs[k * LD + i] = xr[j];
            place(j, Y_K_FAST, k, i);
            ys[k * LD + i] = yr[j];
        }
        __syncthreads();
        if (k0 + KS < depth) fetch(k0 + KS);
        tile_fma(xs, ys, acc, ty, tx);
    }
}

__device__ __forceinline__ void clear(float (&acc)[8][4]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
}

// ----------------------------------------------------------------------------- decays per head
// grid (chunks of the longest sequence, heads, sequences), 128 threads.
__global__ void __launch_bounds__(PT_THREADS) chunk_prepare_head_kernel(const ChunkArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ __align__(16) float xs[KS * LD];
    __shared__ __align__(16) float ys[KS * LD];
    __shared__ double upto[CT];             // sum of g from the chunk's first token up to t
    __shared__ float scale[CT];
    const int head = blockIdx.y, key_head = head / p.heads_per_key;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x);
    if (ck.count <= 0) return;
    if (threadIdx.x < CT) {
        const size_t at = (size_t)(ck.first + threadIdx.x) * p.heads + head;
        const bool in = threadIdx.x < ck.count;
        upto[threadIdx.x] = in ? (double)p.log_decay[at] : 0.0;
        scale[threadIdx.x] = !in ? 0.f : p.v_scale ? p.v_scale[at] : 1.f;
    }
    __syncthreads();
    for (int off = 1; off < CT; off <<= 1) {                        // inclusive sums
        double v = 0.0;
        if (threadIdx.x < CT && threadIdx.x >= off) v = upto[threadIdx.x - off];
        __syncthreads();
        if (threadIdx.x < CT) upto[threadIdx.x] += v;
        __syncthreads();
    }
    if (threadIdx.x < ck.count) {
        const size_t at = (size_t)(ck.first + threadIdx.x) * p.heads + head;
        p.q_from[at] = expf((float)upto[threadIdx.x]) * p.out_scale;
        p.k_to[at] = expf((float)(upto[CT - 1] - upto[threadIdx.x])) * scale[threadIdx.x];
        if (threadIdx.x == 0) p.whole[(size_t)ck.index * p.heads + head] = expf((float)upto[CT - 1]);
    }
    const float* q = p.rows + (size_t)ck.first * p.cols + p.at_q + (size_t)key_head * p.dim;
    const float* k = p.rows + (size_t)ck.first * p.cols + p.at_k + (size_t)key_head * p.dim;
    float acc[8][4];                        // rows s, columns t
    clear(acc);
    tile_product<true, true>(p.dim, [&](int n, int s) { return s < ck.count ? k[(size_t)s * p.cols + n] : 0.f; },
                             [&](int n, int t) { return t < ck.count ? q[(size_t)t * p.cols + n] : 0.f; }, acc, xs, ys);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float* within = p.within + ((size_t)ck.index * p.heads + head) * CT * CT;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int s = 8 * ty + i;
        float v[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = 4 * tx + j;
            v[j] = s <= t && t < ck.count ? acc[i][j] * expf((float)(upto[t] - upto[s])) * scale[s] * p.out_scale : 0.f;
        }
        *reinterpret_cast<float4*>(within + s * CT + 4 * tx) = make_float4(v[0], v[1], v[2], v[3]);
    }
}

// ----------------------------------------------------------------------------- what a chunk writes
// grid (chunks x tiles of the state, heads, sequences), 128 threads: states[m][n] = sum_s v_s[m] k_s[n].
template <bool PER_CHANNEL>
__global__ void __launch_bounds__(PT_THREADS) chunk_write_kernel(const ChunkArgs p, int tiles_n, int tiles) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ __align__(16) float xs[KS * LD];
    __shared__ __align__(16) float ys[KS * LD];
    const int head = blockIdx.y, key_head = head / p.heads_per_key;
    const int which = blockIdx.x % tiles, m0 = which / tiles_n * TILE, n0 = which % tiles_n * TILE;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x / tiles);
    if (ck.count <= 0) return;
    const float* v = p.rows + (size_t)ck.first * p.cols + p.at_v + (size_t)head * p.vdim + m0;
    const float* factor = p.k_to + (size_t)ck.first * p.heads + head;                               // per head: one per token
    const float* k = PER_CHANNEL ? p.k_to + ((size_t)ck.first * p.heads + head) * p.dim + n0
                                 : p.rows + (size_t)ck.first * p.cols + p.at_k + (size_t)key_head * p.dim + n0;
    const size_t k_row = PER_CHANNEL ? (size_t)p.heads * p.dim : (size_t)p.cols;
    const float* scale = PER_CHANNEL && p.v_scale ? p.v_scale + (size_t)ck.first * p.heads + head : nullptr;
    float acc[8][4];
    clear(acc);
    tile_product<false, false>(ck.count,
        [&](int s, int i) {
            if (m0 + i >= p.vdim) return 0.f;
            const float x = v[(size_t)s * p.cols + i];
            return PER_CHANNEL ? (scale ? x * scale[(size_t)s * p.heads] : x) : x * factor[(size_t)s * p.heads];
        },
        [&](int s, int i) { return n0 + i < p.dim ? k[(size_t)s * k_row + i] : 0.f; }, acc, xs, ys);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float* dst = p.states + ((size_t)ck.index * p.heads + head) * p.vdim * p.dim;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int m = m0 + 8 * ty + i;
        if (m >= p.vdim) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (n0 + 4 * tx + j < p.dim) dst[(size_t)m * p.dim + n0 + 4 * tx + j] = acc[i][j];
    }
}

// ----------------------------------------------------------------------------- from chunk to chunk
// grid (blocks of 256 V elements of a head's state, heads, sequences); V: elements a thread moves at once (4 where rows allow).
constexpr int PASS_AHEAD = 8;

template <int V> struct Pack { float v[V]; };
template <int V> __device__ __forceinline__ Pack<V> load_pack(const float* p) {
    Pack<V> r;
    if constexpr (V == 4) { const float4 x = *reinterpret_cast<const float4*>(p); r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w; }
    else r.v[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ void store_pack(float* p, const Pack<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}

template <bool PER_CHANNEL, int V>
__global__ void __launch_bounds__(256) chunk_pass_kernel(const ChunkArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    const int head = blockIdx.y, seq = blockIdx.z, size = p.vdim * p.dim;
    const int e = (blockIdx.x * 256 + threadIdx.x) * V;
    const int begin = p.seq_start[seq], count = p.seq_start[seq + 1] - begin;
    if (count <= 0 || e >= size) return;
    const int chunks = (count + CT - 1) / CT, first = begin / CT + seq;
    float* kept = p.state + ((size_t)p.slots[seq] * p.heads + head) * size + e;
    float* scratch = p.states + ((size_t)first * p.heads + head) * size + e;
    const size_t stride = (size_t)p.heads * size;
    const float* whole = p.whole + ((size_t)first * p.heads + head) * (PER_CHANNEL ? p.dim : 1) + (PER_CHANNEL ? e % p.dim : 0);
    const size_t whole_stride = (size_t)p.heads * (PER_CHANNEL ? p.dim : 1);
    Pack<V> s = load_pack<V>(kept);
    for (int c0 = 0; c0 < chunks; c0 += PASS_AHEAD) {
        Pack<V> d[PASS_AHEAD], f[PASS_AHEAD];
#pragma unroll
        for (int j = 0; j < PASS_AHEAD; ++j) {
            const int c = min(c0 + j, chunks - 1);
            d[j] = load_pack<V>(scratch + c * stride);
            if (PER_CHANNEL) f[j] = load_pack<V>(whole + c * whole_stride);
            else f[j].v[0] = whole[c * whole_stride];
        }
#pragma unroll
        for (int j = 0; j < PASS_AHEAD; ++j) {
            if (c0 + j >= chunks) break;
            store_pack<V>(scratch + (c0 + j) * stride, s);
#pragma unroll
            for (int i = 0; i < V; ++i) s.v[i] = fmaf(f[j].v[PER_CHANNEL ? i : 0], s.v[i], d[j].v[i]);
        }
    }
    store_pack<V>(kept, s);
}

// ----------------------------------------------------------------------------- what a chunk reads
// grid (chunks x tiles of value columns, heads, sequences), 128 threads: out[t][m].
template <bool PER_CHANNEL>
__global__ void __launch_bounds__(PT_THREADS) chunk_read_kernel(const ChunkArgs p, int tiles) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ __align__(16) float xs[KS * LD];
    __shared__ __align__(16) float ys[KS * LD];
    const int head = blockIdx.y, key_head = head / p.heads_per_key, m0 = blockIdx.x % tiles * TILE;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x / tiles);
    if (ck.count <= 0) return;
    const float* q = PER_CHANNEL ? p.q_from + ((size_t)ck.first * p.heads + head) * p.dim
                                 : p.rows + (size_t)ck.first * p.cols + p.at_q + (size_t)key_head * p.dim;
    const size_t q_row = PER_CHANNEL ? (size_t)p.heads * p.dim : (size_t)p.cols;
    const float* states = p.states + (((size_t)ck.index * p.heads + head) * p.vdim + m0) * p.dim;
    const float* within = p.within + ((size_t)ck.index * p.heads + head) * CT * CT;
    const float* v = p.rows + (size_t)ck.first * p.cols + p.at_v + (size_t)head * p.vdim + m0;
    const float* scale = PER_CHANNEL && p.v_scale ? p.v_scale + (size_t)ck.first * p.heads + head : nullptr;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[8][4];
    clear(acc);
    tile_product<true, true>(p.dim, [&](int n, int t) { return t < ck.count ? q[(size_t)t * q_row + n] : 0.f; },
                             [&](int n, int i) { return m0 + i < p.vdim ? states[(size_t)i * p.dim + n] : 0.f; }, acc, xs, ys);
    if (!PER_CHANNEL) {
        const float* factor = p.q_from + (size_t)ck.first * p.heads + head;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float f = 8 * ty + i < ck.count ? factor[(size_t)(8 * ty + i) * p.heads] : 0.f;
            acc[i][0] *= f; acc[i][1] *= f; acc[i][2] *= f; acc[i][3] *= f;
        }
    }
    tile_product<false, false>(ck.count, [&](int s, int t) { return within[s * CT + t]; },
        [&](int s, int i) {
            if (m0 + i >= p.vdim) return 0.f;
            const float x = v[(size_t)s * p.cols + i];
            return scale ? x * scale[(size_t)s * p.heads] : x;
        }, acc, xs, ys);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = 8 * ty + i;
        if (t >= ck.count) continue;
        float* dst = p.out + ((size_t)(ck.first + t) * p.heads + head) * p.vdim + m0 + 4 * tx;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (m0 + 4 * tx + j < p.vdim) dst[j] = acc[i][j];
    }
}

template <bool PER_CHANNEL>
int run_chunks(const ChunkArgs& p, int n_seqs, int chunks, cudaStream_t s) {
    if (PER_CHANNEL) {
        const size_t smem = ((size_t)3 * CT * (p.dim + 4) + (size_t)CT * (CT + 1) + (size_t)7 * p.dim) * sizeof(float);
        static bool configured = false;
        if (!configured) {
            cudaError_t err = cudaFuncSetAttribute(chunk_prepare_channel_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
            if (err != cudaSuccess) QT_FAIL(QT_ERR_LAUNCH, "chunk_prepare: cannot raise shared memory: %s", cudaGetErrorString(err));
            configured = true;
        }
        QT_REQUIRE(smem <= 227 * 1024, "decayed_attention_chunked: %d key channels need more shared memory than a block has", p.dim);
        launch_kernel(chunk_prepare_channel_kernel, dim3(chunks, p.heads, n_seqs), dim3(256), smem, s, p);
    } else {
        launch_kernel(chunk_prepare_head_kernel, dim3(chunks, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p);
    }
    QT_CHECK_LAUNCH("chunk_prepare");
    const int tiles_m = (p.vdim + TILE - 1) / TILE, tiles_n = (p.dim + TILE - 1) / TILE;
    launch_kernel(chunk_write_kernel<PER_CHANNEL>, dim3(chunks * tiles_m * tiles_n, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, tiles_n, tiles_m * tiles_n);
    QT_CHECK_LAUNCH("chunk_write");
    const int size = p.vdim * p.dim;
    const bool wide = p.dim % 4 == 0 && (uintptr_t)p.state % 16 == 0 && (uintptr_t)p.states % 16 == 0 && (uintptr_t)p.whole % 16 == 0;
    if (wide) launch_kernel(chunk_pass_kernel<PER_CHANNEL, 4>, dim3((size + 1023) / 1024, p.heads, n_seqs), dim3(256), 0, s, p);
    else launch_kernel(chunk_pass_kernel<PER_CHANNEL, 1>, dim3((size + 255) / 256, p.heads, n_seqs), dim3(256), 0, s, p);
    QT_CHECK_LAUNCH("chunk_pass");
    launch_kernel(chunk_read_kernel<PER_CHANNEL>, dim3(chunks * tiles_m, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, tiles_m);
    QT_CHECK_LAUNCH("chunk_read");
    return QT_OK;
}

}  // namespace

// The same recurrence, operands and result as qt_decayed_attention_steps (rows: one finished plane).  Scratch of the caller, with
// chunks = T / 64 + n_seqs: states [chunks, heads, vdim, dim], within [chunks, heads, 64, 64], whole [chunks, heads, dim], and q_from and
// k_to [T, heads, dim] (per_channel), or whole [chunks, heads] and q_from, k_to [T, heads].  max_tokens: the most tokens any sequence has.
extern "C" int qt_decayed_attention_chunked(const float* rows, int cols, int at_q, int at_k, int at_v, const float* log_decay, int per_channel,
                                            const float* v_scale, float out_scale, float* state, float* out, const int* seq_start, const int* slots,
                                            int n_seqs, int max_tokens, int heads, int heads_per_key, int dim, int vdim, float* states, float* within,
                                            float* whole, float* q_from, float* k_to, void* stream) {
    QT_REQUIRE(n_seqs >= 0 && max_tokens >= 0 && heads > 0 && heads_per_key > 0 && heads % heads_per_key == 0 && dim > 0 && vdim > 0,
               "decayed_attention_chunked: bad sizes B=%d H=%d/%d dim=%d vdim=%d", n_seqs, heads, heads_per_key, dim, vdim);
    QT_REQUIRE(at_q >= 0 && at_k >= 0 && at_v >= 0 && at_q + heads / heads_per_key * dim <= cols && at_k + heads / heads_per_key * dim <= cols &&
               at_v + heads * vdim <= cols, "decayed_attention_chunked: q, k or v columns outside the rows' %d", cols);
    QT_REQUIRE(heads <= 65535 && n_seqs <= 65535 && (long long)vdim * dim < (1 << 24), "decayed_attention_chunked: too many heads or sequences for one launch");
    QT_REQUIRE(log_decay && states && within && whole && q_from && k_to && (uintptr_t)within % 16 == 0, "decayed_attention_chunked: scratch or decays missing");
    if (n_seqs == 0 || max_tokens == 0) return QT_OK;
    ChunkArgs p{rows, cols, at_q, at_k, at_v, log_decay, v_scale, out_scale, state, out, seq_start, slots, heads, heads_per_key, dim, vdim,
                states, within, whole, q_from, k_to};
    const int chunks = (max_tokens + CT - 1) / CT;
    return per_channel ? run_chunks<true>(p, n_seqs, chunks, (cudaStream_t)stream) : run_chunks<false>(p, n_seqs, chunks, (cudaStream_t)stream);
}

QT_DEFINE_LAST_ERROR(linear_attention_chunk)
