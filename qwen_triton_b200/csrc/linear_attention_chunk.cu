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
// chunk_write_kernel             sum_s (e^{G(s, end)} k_s) v_s^T of a (chunk, head): a product over its tokens per tile of 64 x 64 or 64 x 128.
// chunk_pass_kernel              walks a sequence's chunks elementwise: puts S_c in the place of what chunk c writes, and the last
//                                state back into the sequence's row.
// chunk_read_kernel              o of a (chunk, head): two products per tile, over the state's rows and over the chunk's tokens.
//
// The chunk c of sequence i has the scratch index seq_start[i] / CT + i + c, which is below T / CT + (sequences) and distinct
// for distinct chunks.  States (and their scratch) are stored transposed, [heads, vdim, dim], as in linear_attention.cu.
#include "common.cuh"

#include <math.h>

#include <initializer_list>

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

// Four consecutive floats from p on, `left` of which exist (zeros beyond); one 16-byte load where `vec` says the address allows it.
__device__ __forceinline__ float4 load4(const float* p, int left, bool vec) {
    if (vec && left >= 4) return __ldg(reinterpret_cast<const float4*>(p));
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (left > 0) v.x = __ldg(p);
    if (left > 1) v.y = __ldg(p + 1);
    if (left > 2) v.z = __ldg(p + 2);
    if (left > 3) v.w = __ldg(p + 3);
    return v;
}
__device__ __forceinline__ void put4(float* p, const float4& v, int left, bool vec) {
    if (vec && left >= 4) { *reinterpret_cast<float4*>(p) = v; return; }
    if (left > 0) p[0] = v.x;
    if (left > 1) p[1] = v.y;
    if (left > 2) p[2] = v.z;
    if (left > 3) p[3] = v.w;
}
__device__ __forceinline__ float4 times(const float4& v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); }

// ----------------------------------------------------------------------------- decays per key channel
// grid (chunks of the longest sequence, heads, sequences), PC_THREADS threads; dynamic shared memory (floats): 3 rows of CT x ld, then 15 dim4,
// with dim4 = dim rounded up to a multiple of 4 and ld = dim4 + 4.
constexpr int PC_THREADS = 512;

__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
    return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, acc))));
}
__device__ __forceinline__ float4 mul4(const float4& a, const float4& b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }

// Sixteen values per lane, summed over the lanes of the warp: lane l gets the sum of value l % 16.
__device__ __forceinline__ float transpose_sum(float (&part)[SUB], int lane) {
#pragma unroll
    for (int half = SUB / 2; half >= 1; half >>= 1) {
        const bool upper = (lane & half) != 0;
#pragma unroll
        for (int j = 0; j < half; ++j) {
            const float give = upper ? part[j] : part[j + half], keep = upper ? part[j + half] : part[j];
            part[j] = keep + __shfl_xor_sync(0xffffffffu, give, half);
        }
    }
    return part[0] + __shfl_xor_sync(0xffffffffu, part[0], 16);
}

__global__ void __launch_bounds__(PC_THREADS, 2) chunk_prepare_channel_kernel(const ChunkArgs p, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const int dim = p.dim, quads = (dim + 3) / 4, dim4 = quads * 4, ld = dim4 + 4, head = blockIdx.y, key_head = head / p.heads_per_key;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x);
    if (ck.count <= 0) return;
    float* qs = sm;                        // [CT][ld] q, later e^{sum of g in its run up to t} q
    float* ks = qs + CT * ld;              // [CT][ld] k, later e^{sum of g in its run behind s} k
    float* as = ks + CT * ld;              // [CT][ld] e^{g}
    float* run = as + CT * ld;             // [RUNS][dim4] sum of g over a run
    float* over = run + RUNS * dim4;       // [3][dim4] e^{run 1}, e^{run 2}, e^{run 1 + run 2}
    float* before = over + 3 * dim4;       // [RUNS][dim4] e^{the runs before}
    float* after = before + RUNS * dim4;   // [RUNS][dim4] e^{the runs behind}
    const float* g = p.log_decay + ((size_t)ck.first * p.heads + head) * dim;
    const size_t g_row = (size_t)p.heads * dim;
    const float* rows = p.rows + (size_t)ck.first * p.cols + (size_t)key_head * dim;
    constexpr int AHEAD = 4;
    for (int i0 = threadIdx.x; i0 < CT * quads; i0 += AHEAD * PC_THREADS) {
        float4 q[AHEAD], k[AHEAD], e[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int i = i0 + j * PC_THREADS, t = i / quads, n = i % quads * 4;
            const int left = i < CT * quads && t < ck.count ? dim - n : 0;
            q[j] = load4(rows + (size_t)t * p.cols + p.at_q + n, left, vec);
            k[j] = load4(rows + (size_t)t * p.cols + p.at_k + n, left, vec);
            e[j] = load4(g + (size_t)t * g_row + n, left, vec);
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int i = i0 + j * PC_THREADS, t = i / quads, n = i % quads * 4;
            if (i >= CT * quads) break;
            *reinterpret_cast<float4*>(qs + t * ld + n) = times(q[j], p.out_scale);
            *reinterpret_cast<float4*>(ks + t * ld + n) = k[j];
            *reinterpret_cast<float4*>(as + t * ld + n) = make_float4(expf(e[j].x), expf(e[j].y), expf(e[j].z), expf(e[j].w));
        }
    }
    __syncthreads();
    float* within = p.within + ((size_t)ck.index * p.heads + head) * CT * CT;      // [s][t]
    // inside a run: a warp takes two neighbouring s; its lanes hold k_s decayed so far, multiplied by e^{g_t} as t goes on
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int s = 2 * warp; s < CT; s += 2 * (PC_THREADS / 32)) {
        const int r0 = s / SUB * SUB;
        float part0[SUB], part1[SUB];
#pragma unroll
        for (int j = 0; j < SUB; ++j) part0[j] = part1[j] = 0.f;
        for (int n = lane; n < dim; n += 32) {
            float w0 = ks[s * ld + n], w1 = ks[(s + 1) * ld + n];
#pragma unroll
            for (int j = 0; j < SUB; ++j) {
                const int t = r0 + j;
                if (t < s) continue;
                const float q = qs[t * ld + n], a = as[t * ld + n];
                if (t > s) w0 *= a;
                part0[j] = fmaf(w0, q, part0[j]);
                if (t > s + 1) w1 *= a;
                if (t > s) part1[j] = fmaf(w1, q, part1[j]);
            }
        }
        const float sum0 = transpose_sum(part0, lane), sum1 = transpose_sum(part1, lane);
        if (lane < SUB) { within[s * CT + r0 + lane] = sum0; within[(s + 1) * CT + r0 + lane] = sum1; }
    }
    __syncthreads();
    // running sums inside the runs, forwards on q and backwards on k
    for (int i = threadIdx.x; i < RUNS * dim4; i += PC_THREADS) {
        const int r = i / dim4, n = i % dim4;
        float v[SUB];
#pragma unroll
        for (int j = 0; j < SUB; ++j) v[j] = n < dim && r * SUB + j < ck.count ? __ldg(g + (size_t)(r * SUB + j) * g_row + n) : 0.f;
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < SUB; ++j) { sum += v[j]; qs[(r * SUB + j) * ld + n] *= expf(sum); }
        run[i] = sum;
        float behind = 0.f;
#pragma unroll
        for (int j = SUB - 1; j >= 0; --j) { ks[(r * SUB + j) * ld + n] *= expf(behind); behind += v[j]; }
    }
    __syncthreads();
    for (int n = threadIdx.x; n < dim4; n += PC_THREADS) {
        const float g0 = run[n], g1 = run[dim4 + n], g2 = run[2 * dim4 + n], g3 = run[3 * dim4 + n];
        over[n] = expf(g1); over[dim4 + n] = expf(g2); over[2 * dim4 + n] = expf(g1 + g2);
        before[n] = 1.f; before[dim4 + n] = expf(g0); before[2 * dim4 + n] = expf(g0 + g1); before[3 * dim4 + n] = expf(g0 + g1 + g2);
        after[n] = expf(g1 + g2 + g3); after[dim4 + n] = expf(g2 + g3); after[2 * dim4 + n] = expf(g3); after[3 * dim4 + n] = 1.f;
        if (n < dim) p.whole[((size_t)ck.index * p.heads + head) * dim + n] = expf(g0 + g1 + g2 + g3);
    }
    __syncthreads();
    // between runs: A of run i against run j < i, two t by two s per thread; and zeros where t lies in an earlier run than s
    for (int item = threadIdx.x; item < 6 * 64; item += PC_THREADS) {
        const int pair = item >> 6, local = item & 63;
        const int i = pair < 1 ? 1 : pair < 3 ? 2 : 3, j = pair < 1 ? 0 : pair < 3 ? pair - 1 : pair - 3;
        const int t = i * SUB + (local & 7) * 2, s = j * SUB + (local >> 3) * 2;
        const float* mid = i - j == 3 ? over + 2 * dim4 : i - j == 2 ? (j == 0 ? over : over + dim4) : nullptr;
        float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
        const float *q0 = qs + t * ld, *k0 = ks + s * ld;
        for (int n = 0; n < dim4; n += 4) {
            float4 x0 = *reinterpret_cast<const float4*>(k0 + n), x1 = *reinterpret_cast<const float4*>(k0 + ld + n);
            const float4 y0 = *reinterpret_cast<const float4*>(q0 + n), y1 = *reinterpret_cast<const float4*>(q0 + ld + n);
            if (mid) { const float4 m = *reinterpret_cast<const float4*>(mid + n); x0 = mul4(x0, m); x1 = mul4(x1, m); }
            a00 = dot4(y0, x0, a00); a01 = dot4(y0, x1, a01); a10 = dot4(y1, x0, a10); a11 = dot4(y1, x1, a11);
        }
        *reinterpret_cast<float2*>(within + s * CT + t) = make_float2(a00, a10);
        *reinterpret_cast<float2*>(within + (s + 1) * CT + t) = make_float2(a01, a11);
        const int late = i * SUB + (local >> 3) * 2, early = j * SUB + (local & 7) * 2;
        *reinterpret_cast<float2*>(within + late * CT + early) = make_float2(0.f, 0.f);
        *reinterpret_cast<float2*>(within + (late + 1) * CT + early) = make_float2(0.f, 0.f);
    }
    // the decayed q and k of the whole chunk
    for (int i = threadIdx.x; i < ck.count * quads; i += PC_THREADS) {
        const int t = i / quads, n = i % quads * 4, r = t / SUB;
        const size_t at = ((size_t)(ck.first + t) * p.heads + head) * dim + n;
        put4(p.q_from + at, mul4(*reinterpret_cast<const float4*>(qs + t * ld + n), *reinterpret_cast<const float4*>(before + r * dim4 + n)), dim - n, vec);
        put4(p.k_to + at, mul4(*reinterpret_cast<const float4*>(ks + t * ld + n), *reinterpret_cast<const float4*>(after + r * dim4 + n)), dim - n, vec);
    }
}

// ----------------------------------------------------------------------------- tiles of products
// A block of PT_THREADS threads forms 64 x TN results (TN 64 or 128); thread (ty, tx) of 8 x 16 owns rows 8 ty .. + 7 and the columns
// 4 tx .. + 3 of every 64.  The two operands pass through shared memory in slices of KS rows along the sum.  Results are kept
// as pairs of neighbouring columns: one instruction multiplies and adds both (fma.rn.f32x2, two ordinary float operations).
constexpr int TILE = 64, KS = 16, PT_THREADS = 128;

__device__ __forceinline__ unsigned long long pair_of(float a, float b) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpair(unsigned long long v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ void fma_pair(unsigned long long& d, unsigned long long a, unsigned long long b) {
    asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(d) : "l"(a), "l"(b));
}

template <int TN> struct Acc {
    unsigned long long v[8][TN / 32];      // column pairs: 2 (p % 2) + 64 (p / 2) + 4 tx for pair p
    __device__ __forceinline__ void clear() {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < TN / 32; ++j) v[i][j] = 0ull;
    }
    __device__ __forceinline__ float4 quad(int i, int group) const {
        const float2 a = unpair(v[i][2 * group]), b = unpair(v[i][2 * group + 1]);
        return make_float4(a.x, a.y, b.x, b.y);
    }
    __device__ __forceinline__ void scale_row(int i, float f) {
#pragma unroll
        for (int j = 0; j < TN / 32; ++j) { const float2 a = unpair(v[i][j]); v[i][j] = pair_of(a.x * f, a.y * f); }
    }
};

template <int TN> __device__ __forceinline__ void tile_fma(const float* xs, const float* ys, Acc<TN>& acc, int ty, int tx) {
    constexpr int LDX = TILE + 4, LDY = TN + 4;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
        const float4 a0 = *reinterpret_cast<const float4*>(xs + k * LDX + 8 * ty), a1 = *reinterpret_cast<const float4*>(xs + k * LDX + 8 * ty + 4);
        unsigned long long b[TN / 32];
#pragma unroll
        for (int j = 0; j < TN / 64; ++j) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(ys + k * LDY + 64 * j + 4 * tx);
            b[2 * j] = v.x; b[2 * j + 1] = v.y;
        }
        const float a[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const unsigned long long aa = pair_of(a[i], a[i]);
#pragma unroll
            for (int j = 0; j < TN / 32; ++j) fma_pair(acc.v[i][j], aa, b[j]);
        }
    }
}

// acc += sum over k < depth of x(k, i) y(k, n).  x and y return four neighbouring elements as they lie in memory (zeros outside):
// along k for a K_FAST operand (element (k .. k + 3, i)), else along i.  The next slice is fetched under the arithmetic.
template <int TN, bool X_K_FAST, bool Y_K_FAST, typename FX, typename FY>
__device__ __forceinline__ void tile_product(int depth, FX x, FY y, Acc<TN>& acc, float* xs, float* ys) {
    constexpr int LDX = TILE + 4, LDY = TN + 4, NX = TILE * KS / 4 / PT_THREADS, NY = TN * KS / 4 / PT_THREADS;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float4 xr[NX], yr[NY];
    auto fetch = [&](int k0) {
#pragma unroll
        for (int j = 0; j < NX; ++j) {
            const int e = threadIdx.x + j * PT_THREADS;
            xr[j] = X_K_FAST ? x(k0 + 4 * (e % (KS / 4)), e / (KS / 4)) : x(k0 + e / (TILE / 4), 4 * (e % (TILE / 4)));
        }
#pragma unroll
        for (int j = 0; j < NY; ++j) {
            const int e = threadIdx.x + j * PT_THREADS;
            yr[j] = Y_K_FAST ? y(k0 + 4 * (e % (KS / 4)), e / (KS / 4)) : y(k0 + e / (TN / 4), 4 * (e % (TN / 4)));
        }
    };
    auto place = [&](float* dst, int ld, const float4& v, bool k_fast, int e, int width) {
        if (k_fast) {
            const int k = 4 * (e % (KS / 4)), i = e / (KS / 4);
            dst[k * ld + i] = v.x; dst[(k + 1) * ld + i] = v.y; dst[(k + 2) * ld + i] = v.z; dst[(k + 3) * ld + i] = v.w;
        } else {
            *reinterpret_cast<float4*>(dst + (e / (width / 4)) * ld + 4 * (e % (width / 4))) = v;
        }
    };
    fetch(0);
    for (int k0 = 0; k0 < depth; k0 += KS) {
        __syncthreads();
#pragma unroll
        for (int j = 0; j < NX; ++j) place(xs, LDX, xr[j], X_K_FAST, threadIdx.x + j * PT_THREADS, TILE);
#pragma unroll
        for (int j = 0; j < NY; ++j) place(ys, LDY, yr[j], Y_K_FAST, threadIdx.x + j * PT_THREADS, TN);
        __syncthreads();
        if (k0 + KS < depth) fetch(k0 + KS);
        tile_fma<TN>(xs, ys, acc, ty, tx);
    }
}

// ----------------------------------------------------------------------------- decays per head
// grid (chunks of the longest sequence, heads, sequences), 128 threads.
__global__ void __launch_bounds__(PT_THREADS) chunk_prepare_head_kernel(const ChunkArgs p, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ __align__(16) float xs[KS * (TILE + 4)];
    __shared__ __align__(16) float ys[KS * (TILE + 4)];
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
    Acc<TILE> acc;                          // rows s, columns t
    acc.clear();
    tile_product<TILE, true, true>(p.dim, [&](int n, int s) { return load4(k + (size_t)s * p.cols + n, s < ck.count ? p.dim - n : 0, vec); },
                                   [&](int n, int t) { return load4(q + (size_t)t * p.cols + n, t < ck.count ? p.dim - n : 0, vec); }, acc, xs, ys);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float* within = p.within + ((size_t)ck.index * p.heads + head) * CT * CT;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int s = 8 * ty + i;
        const float4 x = acc.quad(i, 0);
        float v[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = 4 * tx + j;
            v[j] = s <= t && t < ck.count ? v[j] * expf((float)(upto[t] - upto[s])) * scale[s] * p.out_scale : 0.f;
        }
        *reinterpret_cast<float4*>(within + s * CT + 4 * tx) = make_float4(v[0], v[1], v[2], v[3]);
    }
}

// ----------------------------------------------------------------------------- what a chunk writes
// grid (chunks x tiles of the state, heads, sequences), 128 threads: states[m][n] = sum_s v_s[m] k_s[n].
template <bool PER_CHANNEL, int TN>
__global__ void __launch_bounds__(PT_THREADS) chunk_write_kernel(const ChunkArgs p, int tiles_n, int tiles, int vec_v, int vec_k, int vec_s) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ __align__(16) float xs[KS * (TILE + 4)];
    __shared__ __align__(16) float ys[KS * (TN + 4)];
    const int head = blockIdx.y, key_head = head / p.heads_per_key;
    const int which = blockIdx.x % tiles, m0 = which / tiles_n * TILE, n0 = which % tiles_n * TN;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x / tiles);
    if (ck.count <= 0) return;
    const float* v = p.rows + (size_t)ck.first * p.cols + p.at_v + (size_t)head * p.vdim + m0;
    const float* factor = PER_CHANNEL ? (p.v_scale ? p.v_scale + (size_t)ck.first * p.heads + head : nullptr)      // one number per token
                                      : p.k_to + (size_t)ck.first * p.heads + head;
    const float* k = PER_CHANNEL ? p.k_to + ((size_t)ck.first * p.heads + head) * p.dim + n0
                                 : p.rows + (size_t)ck.first * p.cols + p.at_k + (size_t)key_head * p.dim + n0;
    const size_t k_row = PER_CHANNEL ? (size_t)p.heads * p.dim : (size_t)p.cols;
    Acc<TN> acc;
    acc.clear();
    tile_product<TN, false, false>(ck.count,
        [&](int s, int i) {
            const float4 x = load4(v + (size_t)s * p.cols + i, s < ck.count ? p.vdim - m0 - i : 0, vec_v);
            return factor && s < ck.count ? times(x, __ldg(factor + (size_t)s * p.heads)) : x;
        },
        [&](int s, int i) { return load4(k + (size_t)s * k_row + i, s < ck.count ? p.dim - n0 - i : 0, vec_k); }, acc, xs, ys);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float* dst = p.states + ((size_t)ck.index * p.heads + head) * p.vdim * p.dim;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int m = m0 + 8 * ty + i;
        if (m >= p.vdim) continue;
#pragma unroll
        for (int j = 0; j < TN / 64; ++j) {
            const int n = n0 + 64 * j + 4 * tx;
            put4(dst + (size_t)m * p.dim + n, acc.quad(i, j), p.dim - n, vec_s);
        }
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
template <bool PER_CHANNEL, int TN>
__global__ void __launch_bounds__(PT_THREADS) chunk_read_kernel(const ChunkArgs p, int tiles, int vec_q, int vec_v, int vec_s, int vec_o) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ __align__(16) float xs[KS * (TILE + 4)];
    __shared__ __align__(16) float ys[KS * (TN + 4)];
    const int head = blockIdx.y, key_head = head / p.heads_per_key, m0 = blockIdx.x % tiles * TN;
    const Chunk ck = chunk_of(p, blockIdx.z, blockIdx.x / tiles);
    if (ck.count <= 0) return;
    const float* q = PER_CHANNEL ? p.q_from + ((size_t)ck.first * p.heads + head) * p.dim
                                 : p.rows + (size_t)ck.first * p.cols + p.at_q + (size_t)key_head * p.dim;
    const size_t q_row = PER_CHANNEL ? (size_t)p.heads * p.dim : (size_t)p.cols;
    const float* states = p.states + (((size_t)ck.index * p.heads + head) * p.vdim + m0) * p.dim;
    const float* within = p.within + ((size_t)ck.index * p.heads + head) * CT * CT;
    const float* v = p.rows + (size_t)ck.first * p.cols + p.at_v + (size_t)head * p.vdim + m0;
    const float* factor = PER_CHANNEL && p.v_scale ? p.v_scale + (size_t)ck.first * p.heads + head : nullptr;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    Acc<TN> acc;
    acc.clear();
    tile_product<TN, true, true>(p.dim, [&](int n, int t) { return load4(q + (size_t)t * q_row + n, t < ck.count ? p.dim - n : 0, vec_q); },
                                 [&](int n, int i) { return load4(states + (size_t)i * p.dim + n, m0 + i < p.vdim ? p.dim - n : 0, vec_s); }, acc, xs, ys);
    if (!PER_CHANNEL) {
        const float* from = p.q_from + (size_t)ck.first * p.heads + head;
#pragma unroll
        for (int i = 0; i < 8; ++i) acc.scale_row(i, 8 * ty + i < ck.count ? from[(size_t)(8 * ty + i) * p.heads] : 0.f);
    }
    tile_product<TN, false, false>(ck.count, [&](int s, int t) { return load4(within + s * CT + t, s < ck.count ? 4 : 0, true); },
        [&](int s, int i) {
            const float4 x = load4(v + (size_t)s * p.cols + i, s < ck.count ? p.vdim - m0 - i : 0, vec_v);
            return factor && s < ck.count ? times(x, __ldg(factor + (size_t)s * p.heads)) : x;
        }, acc, xs, ys);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = 8 * ty + i;
        if (t >= ck.count) continue;
        float* dst = p.out + ((size_t)(ck.first + t) * p.heads + head) * p.vdim;
#pragma unroll
        for (int j = 0; j < TN / 64; ++j) {
            const int m = m0 + 64 * j + 4 * tx;
            put4(dst + m, acc.quad(i, j), p.vdim - m, vec_o);
        }
    }
}

bool aligned4(const void* p, std::initializer_list<int> strides) {
    bool ok = (uintptr_t)p % 16 == 0;
    for (int s : strides) ok = ok && s % 4 == 0;
    return ok;
}

template <bool PER_CHANNEL>
int run_chunks(const ChunkArgs& p, int n_seqs, int chunks, cudaStream_t s) {
    // 16-byte accesses where the operand's rows start on 16-byte boundaries
    const int vec_v = aligned4(p.rows, {p.cols, p.at_v, p.vdim}), vec_s = aligned4(p.states, {p.dim}), vec_o = aligned4(p.out, {p.vdim});
    const int raw_q = aligned4(p.rows, {p.cols, p.at_q, p.dim}), raw_k = aligned4(p.rows, {p.cols, p.at_k, p.dim});
    const int vec_q = PER_CHANNEL ? aligned4(p.q_from, {p.dim}) : raw_q, vec_k = PER_CHANNEL ? aligned4(p.k_to, {p.dim}) : raw_k;
    if (PER_CHANNEL) {
        const int dim4 = (p.dim + 3) / 4 * 4;
        const size_t smem = ((size_t)3 * CT * (dim4 + 4) + (size_t)(4 + 3 + 8) * dim4) * sizeof(float);
        static bool configured = false;
        if (!configured) {
            cudaError_t err = cudaFuncSetAttribute(chunk_prepare_channel_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
            if (err != cudaSuccess) QT_FAIL(QT_ERR_LAUNCH, "chunk_prepare: cannot raise shared memory: %s", cudaGetErrorString(err));
            configured = true;
        }
        QT_REQUIRE(smem <= 227 * 1024, "decayed_attention_chunked: %d key channels need more shared memory than a block has", p.dim);
        const int vec = raw_q && raw_k && vec_q && vec_k && aligned4(p.log_decay, {p.dim});
        launch_kernel(chunk_prepare_channel_kernel, dim3(chunks, p.heads, n_seqs), dim3(PC_THREADS), smem, s, p, vec);
    } else {
        launch_kernel(chunk_prepare_head_kernel, dim3(chunks, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, (int)(raw_q && raw_k));
    }
    QT_CHECK_LAUNCH("chunk_prepare");
    const int tiles_m = (p.vdim + TILE - 1) / TILE;
    if (p.dim > 64) {
        const int tiles_n = (p.dim + 127) / 128;
        launch_kernel(chunk_write_kernel<PER_CHANNEL, 128>, dim3(chunks * tiles_m * tiles_n, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, tiles_n, tiles_m * tiles_n,
                      vec_v, vec_k, vec_s);
    } else {
        launch_kernel(chunk_write_kernel<PER_CHANNEL, 64>, dim3(chunks * tiles_m, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, 1, tiles_m, vec_v, vec_k, vec_s);
    }
    QT_CHECK_LAUNCH("chunk_write");
    const int size = p.vdim * p.dim;
    const bool wide = vec_s && aligned4(p.state, {}) && aligned4(p.whole, {});
    if (wide) launch_kernel(chunk_pass_kernel<PER_CHANNEL, 4>, dim3((size + 1023) / 1024, p.heads, n_seqs), dim3(256), 0, s, p);
    else launch_kernel(chunk_pass_kernel<PER_CHANNEL, 1>, dim3((size + 255) / 256, p.heads, n_seqs), dim3(256), 0, s, p);
    QT_CHECK_LAUNCH("chunk_pass");
    if (p.vdim > 64) {
        const int tiles = (p.vdim + 127) / 128;
        launch_kernel(chunk_read_kernel<PER_CHANNEL, 128>, dim3(chunks * tiles, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, tiles, vec_q, vec_v, vec_s, vec_o);
    } else {
        launch_kernel(chunk_read_kernel<PER_CHANNEL, 64>, dim3(chunks, p.heads, n_seqs), dim3(PT_THREADS), 0, s, p, 1, vec_q, vec_v, vec_s, vec_o);
    }
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
