// Linear attention with a constant decay per head, and the norm and gate behind it.
//
// Per head a float state S [dim, vdim] is carried from token to token of a sequence:
//     S <- decay_h * S + k_t v_t^T;      o_t = S^T q_t        (o_t is read after token t has been written)
// q, k [heads, dim] and v [heads, vdim] are columns of one projection's float sums (split-K partial sums are added in
// their order); with `act` they pass SiLU on the way in.  The recurrence, the state and the output are float.
//
// linear_attention_scan_kernel   grid (column blocks, heads, sequences): a block owns 32 (or 16) columns of a
//   head's state, a column belongs to 8 neighbouring lanes, each holding RPL consecutive rows of it in registers, so a
//   token costs a thread 2 RPL fused multiply-adds and the column's sum over rows three shuffles.  The state is kept
//   transposed, [slots, heads, vdim, dim], so that the 8 lanes of a column read and write 8 RPL consecutive floats.
//   A sequence's tokens are walked in order, 16 at a time through shared memory; a one-token step is the same kernel
//   with one token, whose cost is the state's bytes.
// linear_attention_step_kernel   few tokens a sequence; it also takes decays that depend on the token, per head or per key
//   channel, a factor on v and q/k heads shared by several heads (qt_decayed_attention_steps).
// group_gate_norm_kernel   out = o / sqrt(mean(o^2) + eps) * weight * gate, the mean over the whole row or over equal parts of it,
//   the gate (sigmoid or SiLU of projection columns) behind the norm or ahead of it, with an optional skip term; rounded
//   once to the output type.
#include "common.cuh"

#include <math.h>
#include <stdlib.h>

using namespace qt;

constexpr int LA_LANES = 8;        // lanes per state column
constexpr int LA_CHUNK = 16;       // tokens staged in shared memory at a time

struct LinAttnParams {
    const float* proj; int n_splits; size_t split_stride; int proj_cols;   // [splits, T, proj_cols]
    int at_q, at_k, at_v;              // first columns of q, k and v
    const float* decay;                // [heads]
    float* state;                      // [slots + 1, heads, vdim, dim]
    float* out;                        // [T, heads, vdim]
    const int* seq_start; const int* slots;
    int heads, dim, vdim, act;
    // decays that depend on the token (null: the constant ones): their logarithms, [T, heads] or [T, heads, dim]
    const float* log_decay;
    const float* v_scale;              // [T, heads] or null: a factor on the token's v
    int heads_per_key;                 // heads that share a q and k head
    float out_scale;                   // factor on o
};
constexpr int LA_CONSTANT = 0, LA_PER_HEAD = 1, LA_PER_CHANNEL = 2;      // what a decay depends on besides its head

__device__ __forceinline__ float la_raw(const LinAttnParams& p, size_t index) {
    float x = __ldg(p.proj + index);
    for (int s = 1; s < p.n_splits; ++s) x += __ldg(p.proj + index + (size_t)s * p.split_stride);
    return x;
}
__device__ __forceinline__ float la_act(const LinAttnParams& p, float x) { return p.act ? x / (1.f + expf(-x)) : x; }

// out[t, c] = SiLU(sum_s proj[s][t, c]) (or the sum itself) for the first `cols` columns of every row: q, k and v of a
// step, summed and activated once where every block of the recurrence would otherwise activate its head's q and k again.
__global__ void linear_attention_prepare_kernel(const float* __restrict__ proj, int n_splits, size_t split_stride, int proj_cols, int cols,
                                                float* __restrict__ out, long long total, int act) {
    pdl_launch_dependents();
    pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const size_t at = (size_t)(i / cols) * proj_cols + (size_t)(i % cols);
        float x = proj[at];
        for (int s = 1; s < n_splits; ++s) x += proj[at + (size_t)s * split_stride];
        out[i] = act ? x / (1.f + expf(-x)) : x;
    }
}

extern "C" int qt_linear_attention_prepare(const float* proj, int n_splits, long long split_stride, int proj_cols, int cols, float* out, int n_tokens,
                                           int act, void* stream) {
    QT_REQUIRE(n_tokens >= 0 && cols > 0 && cols <= proj_cols && n_splits >= 1, "linear_attention_prepare: %d of %d columns", cols, proj_cols);
    if (n_tokens == 0) return QT_OK;
    const long long total = (long long)n_tokens * cols;
    long long blocks = (total + 255) / 256;
    if (blocks > (long long)sm_count() * 16) blocks = (long long)sm_count() * 16;
    launch_kernel(linear_attention_prepare_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, proj, n_splits, (size_t)split_stride, proj_cols,
                  cols, out, total, act);
    QT_CHECK_LAUNCH("linear_attention_prepare");
    return QT_OK;
}

// The same sums for rows whose first `heads` runs of `dim` columns (q heads, then k heads) are rotated by the token's position: in
// each, element i < rd / 2 turns together with element i + rd / 2 by the angle whose cos and sin the table row of the position
// holds (cos | sin, rd columns); the other columns pass.  A thread takes V neighbouring pairs, or V neighbouring columns that
// do not turn; grid (blocks of a row's items, tokens).
template <int V> struct RotPack { float v[V]; };
template <int V> __device__ __forceinline__ RotPack<V> rot_sum(const float* p, int n_splits, size_t stride) {
    RotPack<V> r;
    if constexpr (V == 4) {
        float4 x = __ldg(reinterpret_cast<const float4*>(p));
        for (int s = 1; s < n_splits; ++s) {
            const float4 y = __ldg(reinterpret_cast<const float4*>(p + (size_t)s * stride));
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
        }
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else {
        r.v[0] = __ldg(p);
        for (int s = 1; s < n_splits; ++s) r.v[0] += __ldg(p + (size_t)s * stride);
    }
    return r;
}
template <int V> __device__ __forceinline__ void rot_put(float* p, const RotPack<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}

template <int V>
__global__ void __launch_bounds__(256) linear_attention_rotate_kernel(const float* __restrict__ proj, int n_splits, size_t split_stride, int proj_cols, int cols,
                                                                      float* __restrict__ out, int heads, int dim, int rd, const float* __restrict__ cos_sin,
                                                                      int max_pos, const int* __restrict__ token_pos) {
    pdl_launch_dependents();
    pdl_wait();
    const int item = blockIdx.x * 256 + threadIdx.x, half = rd / 2;
    const int turning = half / V, still = (dim - rd) / V, per_head = turning + still, rotated = heads * per_head;
    if (item >= rotated + (cols - heads * dim) / V) return;
    const size_t t = blockIdx.y;
    const float* row = proj + t * proj_cols;
    float* dst = out + t * cols;
    const int head = item / max(per_head, 1), within = item - head * per_head;
    if (item < rotated && within < turning) {
        const int at = head * dim + within * V;
        const int pos = min(token_pos[t], max_pos - 1);
        const float* table = cos_sin + (size_t)pos * rd + within * V;
        const RotPack<V> c = rot_sum<V>(table, 1, 0), s = rot_sum<V>(table + half, 1, 0);
        const RotPack<V> u = rot_sum<V>(row + at, n_splits, split_stride), w = rot_sum<V>(row + at + half, n_splits, split_stride);
        RotPack<V> a, b;
#pragma unroll
        for (int i = 0; i < V; ++i) {
            a.v[i] = u.v[i] * c.v[i] - w.v[i] * s.v[i];
            b.v[i] = w.v[i] * c.v[i] + u.v[i] * s.v[i];
        }
        rot_put<V>(dst + at, a);
        rot_put<V>(dst + at + half, b);
    } else {
        const int at = item < rotated ? head * dim + rd + (within - turning) * V : heads * dim + (item - rotated) * V;
        rot_put<V>(dst + at, rot_sum<V>(row + at, n_splits, split_stride));
    }
}

extern "C" int qt_linear_attention_rotate(const float* proj, int n_splits, long long split_stride, int proj_cols, int cols, float* out, int n_tokens, int heads,
                                          int dim, int rotary_dim, const float* cos_sin, int max_pos, const int* token_pos, void* stream) {
    QT_REQUIRE(n_tokens >= 0 && cols > 0 && cols <= proj_cols && n_splits >= 1 && heads > 0 && dim > 0 && (long long)heads * dim <= cols,
               "linear_attention_rotate: %d heads of %d in %d of %d columns", heads, dim, cols, proj_cols);
    QT_REQUIRE(rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= dim && cos_sin && max_pos > 0 && token_pos, "linear_attention_rotate: %d of %d elements turn", rotary_dim, dim);
    if (n_tokens == 0) return QT_OK;
    QT_REQUIRE(n_tokens <= 65535, "linear_attention_rotate: %d tokens are too many for one launch", n_tokens);
    const bool wide = rotary_dim % 8 == 0 && dim % 4 == 0 && cols % 4 == 0 && proj_cols % 4 == 0 && split_stride % 4 == 0 && (uintptr_t)proj % 16 == 0 &&
                      (uintptr_t)out % 16 == 0 && (uintptr_t)cos_sin % 16 == 0;
    const int v = wide ? 4 : 1;
    const int items = heads * (dim - rotary_dim / 2) / v + (cols - heads * dim) / v;
    const dim3 grid((items + 255) / 256, n_tokens);
    cudaStream_t s = (cudaStream_t)stream;
    if (wide) launch_kernel(linear_attention_rotate_kernel<4>, grid, dim3(256), 0, s, proj, n_splits, (size_t)split_stride, proj_cols, cols, out, heads, dim, rotary_dim,
                            cos_sin, max_pos, token_pos);
    else launch_kernel(linear_attention_rotate_kernel<1>, grid, dim3(256), 0, s, proj, n_splits, (size_t)split_stride, proj_cols, cols, out, heads, dim, rotary_dim,
                       cos_sin, max_pos, token_pos);
    QT_CHECK_LAUNCH("linear_attention_rotate");
    return QT_OK;
}

// COLS columns of a head's state per block (COLS * 8 threads).  A chunk's q, k and v are fetched into registers while the
// chunk before is worked on (every load of a chunk is issued before the first is used), pass SiLU where asked and go to
// shared memory behind a barrier.
template <int RPL, int COLS>
__global__ void __launch_bounds__(COLS * LA_LANES) linear_attention_scan_kernel(const LinAttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int THREADS = COLS * LA_LANES;
    constexpr int STRIDE = LA_LANES * (RPL + 4);          // a token's q (or k) row in shared memory: 4 floats of padding per lane's
    constexpr int ROW = LA_LANES * RPL;                   // piece, so that the 8 lanes' 16-byte reads fall on different banks
    constexpr int QK_PER = LA_CHUNK * ROW / THREADS;      // q (and k) elements of a chunk per thread
    constexpr int V_PER = LA_CHUNK * COLS / THREADS;      // v elements of a chunk per thread (2)
    __shared__ __align__(16) float qs[LA_CHUNK * STRIDE];
    __shared__ __align__(16) float ks[LA_CHUNK * STRIDE];
    __shared__ float vs[LA_CHUNK * COLS];
    const int head = blockIdx.y, seq = blockIdx.z;
    const int lane = threadIdx.x % LA_LANES, col_in_block = threadIdx.x / LA_LANES;
    const int col = blockIdx.x * COLS + col_in_block;
    const int begin = p.seq_start[seq], end = p.seq_start[seq + 1];
    if (begin >= end) return;
    const float decay = p.decay[head];
    const bool live = col < p.vdim;
    float* state = p.state + (((size_t)p.slots[seq] * p.heads + head) * p.vdim + (live ? col : 0)) * p.dim;
    const int row0 = lane * RPL;
    const bool vec = p.dim % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    float S[RPL];
#pragma unroll
    for (int i = 0; i < RPL; ++i) S[i] = 0.f;
    if (live) {
        if (vec) {
#pragma unroll
            for (int i = 0; i < RPL; i += 4)
                if (row0 + i < p.dim) {
                    const float4 v = *reinterpret_cast<const float4*>(state + row0 + i);
                    S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
                }
        } else {
#pragma unroll
            for (int i = 0; i < RPL; ++i)
                if (row0 + i < p.dim) S[i] = state[row0 + i];
        }
    }
    float qr[QK_PER], kr[QK_PER], vr[V_PER];
    auto fetch = [&](int t0) {                             // the chunk from token t0 on, into registers
        const int count = min(LA_CHUNK, end - t0);
#pragma unroll
        for (int j = 0; j < QK_PER; ++j) {
            const int i = threadIdx.x + j * THREADS, tok = i / ROW, r = i % ROW;
            const bool has = tok < count && r < p.dim;
            const size_t row = (size_t)(t0 + tok) * p.proj_cols + (size_t)head * p.dim + r;
            qr[j] = has ? la_raw(p, row + p.at_q) : 0.f;
            kr[j] = has ? la_raw(p, row + p.at_k) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < V_PER; ++j) {
            const int i = threadIdx.x + j * THREADS, tok = i / COLS, c = blockIdx.x * COLS + i % COLS;
            vr[j] = (tok < count && c < p.vdim) ? la_raw(p, (size_t)(t0 + tok) * p.proj_cols + p.at_v + (size_t)head * p.vdim + c) : 0.f;
        }
    };
    fetch(begin);
    for (int t0 = begin; t0 < end; t0 += LA_CHUNK) {
        const int count = min(LA_CHUNK, end - t0);
        __syncthreads();                                   // the chunk before has been read
#pragma unroll
        for (int j = 0; j < QK_PER; ++j) {
            const int i = threadIdx.x + j * THREADS, tok = i / ROW, r = i % ROW;
            const int at = tok * STRIDE + (r / RPL) * (RPL + 4) + r % RPL;
            qs[at] = la_act(p, qr[j]);
            ks[at] = la_act(p, kr[j]);
        }
#pragma unroll
        for (int j = 0; j < V_PER; ++j) vs[threadIdx.x + j * THREADS] = la_act(p, vr[j]);
        __syncthreads();
        if (t0 + LA_CHUNK < end) fetch(t0 + LA_CHUNK);     // in flight while this chunk is worked on
#pragma unroll 2
        for (int tok = 0; tok < count; ++tok) {
            const float v = vs[tok * COLS + col_in_block];
            const float* qrow = qs + tok * STRIDE + lane * (RPL + 4);
            const float* krow = ks + tok * STRIDE + lane * (RPL + 4);
            float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
            for (int i = 0; i < RPL; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(krow + i);
                const float4 q4 = *reinterpret_cast<const float4*>(qrow + i);
                S[i] = fmaf(decay, S[i], k4.x * v);         a0 = fmaf(S[i], q4.x, a0);
                S[i + 1] = fmaf(decay, S[i + 1], k4.y * v); a1 = fmaf(S[i + 1], q4.y, a1);
                S[i + 2] = fmaf(decay, S[i + 2], k4.z * v); a2 = fmaf(S[i + 2], q4.z, a2);
                S[i + 3] = fmaf(decay, S[i + 3], k4.w * v); a3 = fmaf(S[i + 3], q4.w, a3);
            }
            float acc = (a0 + a1) + (a2 + a3);
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            if (lane == 0 && live) p.out[((size_t)(t0 + tok) * p.heads + head) * p.vdim + col] = acc;
        }
    }
    if (live) {
        if (vec) {
#pragma unroll
            for (int i = 0; i < RPL; i += 4)
                if (row0 + i < p.dim) *reinterpret_cast<float4*>(state + row0 + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
        } else {
#pragma unroll
            for (int i = 0; i < RPL; ++i)
                if (row0 + i < p.dim) state[row0 + i] = S[i];
        }
    }
}

// Steps in which no sequence brings more than a few tokens (one-token steps above all): nothing is staged or fetched
// ahead, a thread reads its rows' q and k from the projection itself (the 32 columns of a block read the same ones, from
// L1), so the kernel is short and light in registers and many blocks share an SM; its cost is the state's bytes.
template <int RPL, int MODE>
__global__ void __launch_bounds__(32 * LA_LANES) linear_attention_step_kernel(const LinAttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int head = blockIdx.y, seq = blockIdx.z;
    const int lane = threadIdx.x % LA_LANES, col = blockIdx.x * 32 + threadIdx.x / LA_LANES;
    const int begin = p.seq_start[seq], end = p.seq_start[seq + 1];
    if (begin >= end) return;
    const float constant = MODE == LA_CONSTANT ? p.decay[head] : 0.f;
    const int key_head = MODE == LA_CONSTANT ? head : head / p.heads_per_key;
    const bool live = col < p.vdim;
    float* state = p.state + (((size_t)p.slots[seq] * p.heads + head) * p.vdim + (live ? col : 0)) * p.dim;
    const int row0 = 4 * lane;                              // this lane holds rows 4 lane + at(i): its 16-byte pieces lie beside its neighbours'
    auto at = [](int i) { return i / 4 * 4 * LA_LANES + i % 4; };
    const bool vec = p.dim % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    float S[RPL];
#pragma unroll
    for (int i = 0; i < RPL; ++i) S[i] = 0.f;
    if (live) {
        if (vec) {
#pragma unroll
            for (int i = 0; i < RPL; i += 4)
                if (row0 + at(i) < p.dim) {
                    const float4 v = *reinterpret_cast<const float4*>(state + row0 + at(i));
                    S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
                }
        } else {
#pragma unroll
            for (int i = 0; i < RPL; ++i)
                if (row0 + at(i) < p.dim) S[i] = state[row0 + at(i)];
        }
    }
    const bool quads = p.n_splits == 1 && p.dim % 4 == 0 && p.at_q % 4 == 0 && p.at_k % 4 == 0 && p.proj_cols % 4 == 0 && ((uintptr_t)p.proj & 15) == 0;
    for (int t = begin; t < end; ++t) {
        const size_t row = (size_t)t * p.proj_cols;
        float v = live ? la_act(p, la_raw(p, row + p.at_v + (size_t)head * p.vdim + col)) : 0.f;
        float decay[MODE == LA_PER_CHANNEL ? RPL : 1];
        decay[0] = constant;
        if (MODE != LA_CONSTANT) {
            const size_t th = (size_t)t * p.heads + head;
            if (p.v_scale) v *= __ldg(p.v_scale + th);
            if (MODE == LA_PER_HEAD) decay[0] = expf(__ldg(p.log_decay + th));
            else if (vec && ((uintptr_t)p.log_decay & 15) == 0) {
#pragma unroll
                for (int i = 0; i < (MODE == LA_PER_CHANNEL ? RPL : 1); i += 4) {
                    const float4 g = row0 + at(i) < p.dim ? __ldg(reinterpret_cast<const float4*>(p.log_decay + th * p.dim + row0 + at(i))) : make_float4(0.f, 0.f, 0.f, 0.f);
                    const float e[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) if (MODE == LA_PER_CHANNEL) decay[(i + j) % (MODE == LA_PER_CHANNEL ? RPL : 1)] = e[j];
                }
            } else {
#pragma unroll
                for (int i = 0; i < (MODE == LA_PER_CHANNEL ? RPL : 1); ++i) decay[i] = row0 + at(i) < p.dim ? __ldg(p.log_decay + th * p.dim + row0 + at(i)) : 0.f;
            }
        }
        float q[RPL], k[RPL];
        const size_t q_at = row + p.at_q + (size_t)key_head * p.dim + row0, k_at = row + p.at_k + (size_t)key_head * p.dim + row0;
        if (quads) {                                        // 16-byte loads of a row that is finished and aligned
#pragma unroll
            for (int i = 0; i < RPL; i += 4) {
                const bool has = row0 + at(i) < p.dim;
                const float4 q4 = has ? __ldg(reinterpret_cast<const float4*>(p.proj + q_at + at(i))) : make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 k4 = has ? __ldg(reinterpret_cast<const float4*>(p.proj + k_at + at(i))) : make_float4(0.f, 0.f, 0.f, 0.f);
                q[i] = q4.x; q[i + 1] = q4.y; q[i + 2] = q4.z; q[i + 3] = q4.w;
                k[i] = k4.x; k[i + 1] = k4.y; k[i + 2] = k4.z; k[i + 3] = k4.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < RPL; ++i) {                 // every load of the token ahead of its arithmetic
                const bool has = row0 + at(i) < p.dim;
                q[i] = has ? la_raw(p, q_at + at(i)) : 0.f;
                k[i] = has ? la_raw(p, k_at + at(i)) : 0.f;
            }
        }
        if (MODE == LA_PER_CHANNEL) {                           // the logarithms are turned once everything has been asked for
#pragma unroll
            for (int i = 0; i < (MODE == LA_PER_CHANNEL ? RPL : 1); ++i) decay[i] = expf(decay[i]);
        }
        float a0 = 0.f, a1 = 0.f;
#pragma unroll
        for (int i = 0; i < RPL; i += 2) {
            S[i] = fmaf(decay[MODE == LA_PER_CHANNEL ? i : 0], S[i], la_act(p, k[i]) * v);             a0 = fmaf(S[i], la_act(p, q[i]), a0);
            S[i + 1] = fmaf(decay[MODE == LA_PER_CHANNEL ? i + 1 : 0], S[i + 1], la_act(p, k[i + 1]) * v); a1 = fmaf(S[i + 1], la_act(p, q[i + 1]), a1);
        }
        float acc = a0 + a1;
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        acc += __shfl_xor_sync(0xffffffffu, acc, 2);
        acc += __shfl_xor_sync(0xffffffffu, acc, 4);
        if (lane == 0 && live) p.out[((size_t)t * p.heads + head) * p.vdim + col] = MODE == LA_CONSTANT ? acc : acc * p.out_scale;
    }
    if (live) {
        if (vec) {
#pragma unroll
            for (int i = 0; i < RPL; i += 4)
                if (row0 + at(i) < p.dim) *reinterpret_cast<float4*>(state + row0 + at(i)) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
        } else {
#pragma unroll
            for (int i = 0; i < RPL; ++i)
                if (row0 + at(i) < p.dim) state[row0 + at(i)] = S[i];
        }
    }
}

// The same recurrence with a whole warp per column, for a step that brings one long portion or few of them: lane l holds the
// column's rows i * 128 + 4 l + e (i < NV, e < 4), so a token is a shorter chain of instructions per warp and an SM holds
// four times the warps, which is what hides a chain's latencies when there are few columns to go round.  Every warp
// reads the whole q and k of a token from shared memory, so this form moves four times the shared-memory bytes of the
// one above: it loses where the blocks of the other form fill the machine.
constexpr int LW_COLS = 8;         // state columns per block, one warp each
constexpr int LW_THREADS = LW_COLS * 32;

template <int NV>
__global__ void __launch_bounds__(LW_THREADS) linear_attention_scan_warp_kernel(const LinAttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int ROW = NV * 128;                         // a token's q (or k) row in shared memory, zeros beyond dim
    constexpr int QK_PER = LA_CHUNK * ROW / LW_THREADS;   // q (and k) elements of a chunk per thread
    __shared__ __align__(16) float qs[LA_CHUNK * ROW];
    __shared__ __align__(16) float ks[LA_CHUNK * ROW];
    __shared__ float vs[LA_CHUNK * LW_COLS];
    const int head = blockIdx.y, seq = blockIdx.z;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int col = blockIdx.x * LW_COLS + warp;
    const int begin = p.seq_start[seq], end = p.seq_start[seq + 1];
    if (begin >= end) return;
    const float decay = p.decay[head];
    const bool live = col < p.vdim;
    float* state = p.state + (((size_t)p.slots[seq] * p.heads + head) * p.vdim + (live ? col : 0)) * p.dim;
    const bool vec = p.dim % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    float S[NV][4];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int r = i * 128 + 4 * lane;
        S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
        if (!live) continue;
        if (vec) {
            if (r < p.dim) { const float4 v = *reinterpret_cast<const float4*>(state + r); S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w; }
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (r + e < p.dim) S[i][e] = state[r + e];
        }
    }
    float qr[QK_PER], kr[QK_PER], vr = 0.f;
    auto fetch = [&](int t0) {                             // the chunk from token t0 on, into registers
        const int count = min(LA_CHUNK, end - t0);
#pragma unroll
        for (int j = 0; j < QK_PER; ++j) {
            const int i = threadIdx.x + j * LW_THREADS, tok = i / ROW, r = i % ROW;
            const bool has = tok < count && r < p.dim;
            const size_t row = (size_t)(t0 + tok) * p.proj_cols + (size_t)head * p.dim + r;
            qr[j] = has ? la_raw(p, row + p.at_q) : 0.f;
            kr[j] = has ? la_raw(p, row + p.at_k) : 0.f;
        }
        if (threadIdx.x < LA_CHUNK * LW_COLS) {
            const int tok = threadIdx.x / LW_COLS, c = blockIdx.x * LW_COLS + threadIdx.x % LW_COLS;
            vr = (tok < count && c < p.vdim) ? la_raw(p, (size_t)(t0 + tok) * p.proj_cols + p.at_v + (size_t)head * p.vdim + c) : 0.f;
        }
    };
    fetch(begin);
    for (int t0 = begin; t0 < end; t0 += LA_CHUNK) {
        const int count = min(LA_CHUNK, end - t0);
        __syncthreads();                                   // the chunk before has been read
#pragma unroll
        for (int j = 0; j < QK_PER; ++j) {
            qs[threadIdx.x + j * LW_THREADS] = la_act(p, qr[j]);
            ks[threadIdx.x + j * LW_THREADS] = la_act(p, kr[j]);
        }
        if (threadIdx.x < LA_CHUNK * LW_COLS) vs[threadIdx.x] = la_act(p, vr);
        __syncthreads();
        if (t0 + LA_CHUNK < end) fetch(t0 + LA_CHUNK);     // in flight while this chunk is worked on
#pragma unroll 4
        for (int tok = 0; tok < count; ++tok) {
            const float v = vs[tok * LW_COLS + warp];
            float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const float4 k4 = *reinterpret_cast<const float4*>(ks + tok * ROW + i * 128 + 4 * lane);
                const float4 q4 = *reinterpret_cast<const float4*>(qs + tok * ROW + i * 128 + 4 * lane);
                S[i][0] = fmaf(decay, S[i][0], k4.x * v); a0 = fmaf(S[i][0], q4.x, a0);
                S[i][1] = fmaf(decay, S[i][1], k4.y * v); a1 = fmaf(S[i][1], q4.y, a1);
                S[i][2] = fmaf(decay, S[i][2], k4.z * v); a2 = fmaf(S[i][2], q4.z, a2);
                S[i][3] = fmaf(decay, S[i][3], k4.w * v); a3 = fmaf(S[i][3], q4.w, a3);
            }
            const float acc = warp_sum((a0 + a1) + (a2 + a3));
            if (lane == 0 && live) p.out[((size_t)(t0 + tok) * p.heads + head) * p.vdim + col] = acc;
        }
    }
    if (!live) return;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int r = i * 128 + 4 * lane;
        if (vec) {
            if (r < p.dim) *reinterpret_cast<float4*>(state + r) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (r + e < p.dim) state[r + e] = S[i][e];
        }
    }
}

extern "C" int qt_linear_attention_scan(const float* proj, int n_splits, long long split_stride, int proj_cols, int at_q, int at_k, int at_v,
                                        const float* decay, float* state, float* out, const int* seq_start, const int* slots, int n_seqs,
                                        int heads, int dim, int vdim, int act, int max_q_len, void* stream) {
    QT_REQUIRE(n_seqs >= 0 && heads > 0 && dim > 0 && vdim > 0 && n_splits >= 1, "linear_attention_scan: bad sizes B=%d H=%d dim=%d vdim=%d", n_seqs, heads, dim, vdim);
    QT_REQUIRE(dim <= LA_LANES * 32, "linear_attention_scan: %d key channels per head are beyond what a column's lanes hold (%d)", dim, LA_LANES * 32);
    QT_REQUIRE(at_q >= 0 && at_k >= 0 && at_v >= 0 && at_q + heads * dim <= proj_cols && at_k + heads * dim <= proj_cols && at_v + heads * vdim <= proj_cols,
               "linear_attention_scan: q, k or v columns outside the projection's %d", proj_cols);
    if (n_seqs == 0) return QT_OK;
    LinAttnParams p{proj, n_splits, (size_t)split_stride, proj_cols, at_q, at_k, at_v, decay, state, out, seq_start, slots, heads, dim, vdim, act,
                    nullptr, nullptr, 1, 1.f};
    cudaStream_t s = (cudaStream_t)stream;
    // blocks of 32 columns where they fill the machine twice over (many sequences: every block stages its head's q and k
    // itself), else of 16, so that one prompt still gives most SMs a block
    const bool wide = (long long)((vdim + 31) / 32) * heads * n_seqs >= 2LL * sm_count();
    if (max_q_len <= 4) {                                  // few tokens a sequence: the short kernel
        const dim3 grid((vdim + 31) / 32, heads, n_seqs), block(32 * LA_LANES);
        if (dim <= LA_LANES * 8) launch_kernel(linear_attention_step_kernel<8, LA_CONSTANT>, grid, block, 0, s, p);
        else if (dim <= LA_LANES * 16) launch_kernel(linear_attention_step_kernel<16, LA_CONSTANT>, grid, block, 0, s, p);
        else launch_kernel(linear_attention_step_kernel<32, LA_CONSTANT>, grid, block, 0, s, p);
        QT_CHECK_LAUNCH("linear_attention_scan");
        return QT_OK;
    }
    // long portions of few sequences, with a head's rows within what 32 lanes hold four at a time: a warp per column
    static const bool warp_form = [] { const char* env = getenv("QT_B200_LINEAR_WARP"); return !(env && env[0] == '0'); }();
    if (warp_form && max_q_len >= 64 && dim > 64 && (long long)((vdim + 15) / 16) * heads * n_seqs < 2LL * sm_count()) {
        const dim3 grid((vdim + LW_COLS - 1) / LW_COLS, heads, n_seqs), block(LW_THREADS);
        if (dim <= 128) launch_kernel(linear_attention_scan_warp_kernel<1>, grid, block, 0, s, p);
        else launch_kernel(linear_attention_scan_warp_kernel<2>, grid, block, 0, s, p);
        QT_CHECK_LAUNCH("linear_attention_scan");
        return QT_OK;
    }
#define QT_LAUNCH_LA(RPL)                                                                                                              \
    do {                                                                                                                               \
        if (wide) launch_kernel(linear_attention_scan_kernel<RPL, 32>, dim3((vdim + 31) / 32, heads, n_seqs), dim3(32 * LA_LANES), 0, s, p); \
        else launch_kernel(linear_attention_scan_kernel<RPL, 16>, dim3((vdim + 15) / 16, heads, n_seqs), dim3(16 * LA_LANES), 0, s, p);      \
    } while (0)
    if (dim <= LA_LANES * 8) QT_LAUNCH_LA(8);
    else if (dim <= LA_LANES * 16) QT_LAUNCH_LA(16);
    else QT_LAUNCH_LA(32);
#undef QT_LAUNCH_LA
    QT_CHECK_LAUNCH("linear_attention_scan");
    return QT_OK;
}

// The recurrence with decays that depend on the token, token by token: S <- diag(exp(log_decay_t)) S + k_t (v_scale_t v_t)^T,
// o_t = out_scale S^T q_t.  log_decay is [T, heads] or (per_channel) [T, heads, dim]; q and k have heads / heads_per_key heads.
// The form for steps of few tokens a sequence (linear_attention_chunk.cu takes long ones).
extern "C" int qt_decayed_attention_steps(const float* proj, int n_splits, long long split_stride, int proj_cols, int at_q, int at_k, int at_v,
                                          const float* log_decay, int per_channel, const float* v_scale, float out_scale, float* state, float* out,
                                          const int* seq_start, const int* slots, int n_seqs, int heads, int heads_per_key, int dim, int vdim,
                                          void* stream) {
    QT_REQUIRE(n_seqs >= 0 && heads > 0 && heads_per_key > 0 && heads % heads_per_key == 0 && dim > 0 && vdim > 0 && n_splits >= 1,
               "decayed_attention: bad sizes B=%d H=%d/%d dim=%d vdim=%d", n_seqs, heads, heads_per_key, dim, vdim);
    QT_REQUIRE(dim <= LA_LANES * 32, "decayed_attention: %d key channels per head are beyond what a column's lanes hold (%d)", dim, LA_LANES * 32);
    QT_REQUIRE(at_q >= 0 && at_k >= 0 && at_v >= 0 && at_q + heads / heads_per_key * dim <= proj_cols && at_k + heads / heads_per_key * dim <= proj_cols &&
               at_v + heads * vdim <= proj_cols, "decayed_attention: q, k or v columns outside the projection's %d", proj_cols);
    QT_REQUIRE(log_decay != nullptr && heads <= 65535 && n_seqs <= 65535, "decayed_attention: no decays, or too many heads or sequences for one launch");
    if (n_seqs == 0) return QT_OK;
    LinAttnParams p{proj, n_splits, (size_t)split_stride, proj_cols, at_q, at_k, at_v, nullptr, state, out, seq_start, slots, heads, dim, vdim, 0,
                    log_decay, v_scale, heads_per_key, out_scale};
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid((vdim + 31) / 32, heads, n_seqs), block(32 * LA_LANES);
#define QT_LAUNCH_STEPS(RPL)                                                                             \
    do {                                                                                                 \
        if (per_channel) launch_kernel(linear_attention_step_kernel<RPL, LA_PER_CHANNEL>, grid, block, 0, s, p); \
        else launch_kernel(linear_attention_step_kernel<RPL, LA_PER_HEAD>, grid, block, 0, s, p);         \
    } while (0)
    if (dim <= LA_LANES * 8) QT_LAUNCH_STEPS(8);
    else if (dim <= LA_LANES * 16) QT_LAUNCH_STEPS(16);
    else QT_LAUNCH_STEPS(32);
#undef QT_LAUNCH_STEPS
    QT_CHECK_LAUNCH("decayed_attention_steps");
    return QT_OK;
}

// ----------------------------------------------------------------------------- skip, gate and norm behind a recurrence
// y = o (+ skip[h] * x, h the head of the element); with gate_first y *= a(g); then y / sqrt(mean(y^2) + eps) * weight * scale over
// `groups` equal parts of the row, each by its own mean; without gate_first times a(g).  a is the sigmoid or (silu) SiLU of the
// gate's sums.  weight has an element per column, or (weight_len = the part's width) one per column of a part.  Rounded once.
struct GroupNormParams {
    const float* o;                                                    // [T, width]
    const float* x; int x_cols, at_x; const float* skip; int per_skip;   // x [T, x_cols] from column at_x; skip[i / per_skip]; or null
    const float* proj; int n_splits; size_t split_stride; int proj_cols, at_gate;    // the gate's sums; or null
    const float* weight; int weight_len;
    float eps, scale;
    int width, part, silu, gate_first;
};

__device__ __forceinline__ float gn_gate_sum(const GroupNormParams& p, size_t t, int i) {
    const float* at = p.proj + t * p.proj_cols + p.at_gate + i;
    float g = 0.f;
    for (int s0 = 0; s0 < p.n_splits; s0 += 8) {                        // eight loads of a split product's planes in flight
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = s0 + j < p.n_splits ? __ldg(at + (size_t)(s0 + j) * p.split_stride) : 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) g += v[j];
    }
    return g;
}
__device__ __forceinline__ float gn_gate_value(const GroupNormParams& p, float g) {
    const float sig = 1.f / (1.f + expf(-g));
    return p.silu ? g * sig : sig;
}
__device__ __forceinline__ float gn_gate(const GroupNormParams& p, size_t t, int i) { return gn_gate_value(p, gn_gate_sum(p, t, i)); }
__device__ __forceinline__ float gn_value(const GroupNormParams& p, size_t t, int i) {
    float y = __ldg(p.o + t * p.width + i);
    if (p.x) y += __ldg(p.skip + i / p.per_skip) * __ldg(p.x + t * p.x_cols + p.at_x + i);
    return y;
}

// WARP: a part per warp (parts of up to 32 GN_CACHE elements), else a part per block (up to GN_CACHE elements a thread); elements
// beyond what the registers hold are formed again in the second pass.  grid (tokens, blocks of parts).
constexpr int GN_CACHE = 8;

// ONE_PLANE: the gate's sums are finished, so a thread asks for everything it needs before it uses the first value.
template <typename TO, bool WARP, bool ONE_PLANE>
__global__ void group_gate_norm_kernel(const GroupNormParams p, TO* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    const int part = WARP ? blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.y;
    if (WARP && part * p.part >= p.width) return;                       // whole warps leave; a block's threads stay together otherwise
    const int first = WARP ? threadIdx.x & 31 : threadIdx.x, step = WARP ? 32 : blockDim.x, base = part * p.part;
    float y[GN_CACHE], gate[GN_CACHE], sq = 0.f;
    const float* o = p.o + t * p.width + base;
    const float* x = p.x ? p.x + t * p.x_cols + p.at_x + base : nullptr;
    const float* g = p.proj ? p.proj + t * p.proj_cols + p.at_gate + base : nullptr;
#pragma unroll
    for (int j = 0; j < GN_CACHE; ++j) {
        const int i = first + j * step;
        const bool in = i < p.part;
        y[j] = in ? __ldg(o + i) : 0.f;
        if (ONE_PLANE) gate[j] = in && g ? __ldg(g + i) : 0.f;
        else gate[j] = in && g ? gn_gate_sum(p, t, base + i) : 0.f;
    }
    if (x) {
#pragma unroll
        for (int j = 0; j < GN_CACHE; ++j) {
            const int i = first + j * step;
            if (i < p.part) y[j] = fmaf(__ldg(p.skip + (base + i) / p.per_skip), __ldg(x + i), y[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < GN_CACHE; ++j) {
        gate[j] = g ? gn_gate_value(p, gate[j]) : 1.f;
        if (p.gate_first) { y[j] *= gate[j]; gate[j] = 1.f; }
        sq += y[j] * y[j];
    }
    for (int i = first + GN_CACHE * step; i < p.part; i += step) {
        const float v = gn_value(p, t, base + i) * (p.proj && p.gate_first ? gn_gate(p, t, base + i) : 1.f);
        sq += v * v;
    }
    const float inv = rsqrtf((WARP ? warp_sum(sq) : block_sum(sq, scratch)) / (float)p.part + p.eps) * p.scale;
    auto finish = [&](float v, int i) { out[t * p.width + base + i] = from_float<TO>(v * inv * __ldg(p.weight + (p.weight_len == p.part ? i : base + i))); };
#pragma unroll
    for (int j = 0; j < GN_CACHE; ++j)
        if (first + j * step < p.part) finish(y[j] * gate[j], first + j * step);
    for (int i = first + GN_CACHE * step; i < p.part; i += step) finish(gn_value(p, t, base + i) * (p.proj ? gn_gate(p, t, base + i) : 1.f), i);
}

extern "C" int qt_group_gate_norm(const float* o, const float* x, int x_cols, int at_x, const float* skip, int skips, const float* proj, int n_splits,
                                  long long split_stride, int proj_cols, int at_gate, const float* weight, int weight_len, float eps, float scale,
                                  int groups, int silu, int gate_first, void* out, int out_dtype, int n_tokens, int width, void* stream) {
    QT_REQUIRE(n_tokens >= 0 && width > 0 && groups > 0 && width % groups == 0 && eps > 0.f, "group_gate_norm: bad sizes T=%d width=%d in %d parts", n_tokens, width, groups);
    QT_REQUIRE(weight_len == width || weight_len == width / groups, "group_gate_norm: a weight of %d for %d columns in %d parts", weight_len, width, groups);
    QT_REQUIRE(!proj || (at_gate >= 0 && at_gate + width <= proj_cols && n_splits >= 1), "group_gate_norm: gate columns outside the projection");
    QT_REQUIRE(!x || (skip && skips > 0 && width % skips == 0 && at_x >= 0 && at_x + width <= x_cols), "group_gate_norm: the skip term's operands do not fit");
    if (n_tokens == 0) return QT_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int part = width / groups;
    GroupNormParams p{o, x, x_cols, at_x, skip, x ? width / skips : 1, proj, n_splits, (size_t)split_stride, proj_cols, at_gate, weight, weight_len, eps, scale,
                      width, part, silu, gate_first};
    return QT_DISPATCH_DTYPE(out_dtype, "group_gate_norm", {
        const bool one = n_splits == 1;
        if (groups > 1 && part <= 32 * GN_CACHE) {
            const dim3 grid(n_tokens, (groups + 3) / 4);
            if (one) launch_kernel(group_gate_norm_kernel<T, true, true>, grid, dim3(128), 0, s, p, (T*)out);
            else launch_kernel(group_gate_norm_kernel<T, true, false>, grid, dim3(128), 0, s, p, (T*)out);
        } else {
            int threads = ((part + GN_CACHE * 32 - 1) / (GN_CACHE * 32)) * 32;      // 8 elements a thread; few tokens: fewer each
            if (n_tokens < 256) threads = ((part + 63) / 64) * 32;
            threads = threads < 64 ? 64 : threads > 1024 ? 1024 : threads;
            if (one) launch_kernel(group_gate_norm_kernel<T, false, true>, dim3(n_tokens, groups), dim3(threads), 0, s, p, (T*)out);
            else launch_kernel(group_gate_norm_kernel<T, false, false>, dim3(n_tokens, groups), dim3(threads), 0, s, p, (T*)out);
        }
        QT_CHECK_LAUNCH("group_gate_norm");
        return QT_OK;
    });
}

QT_DEFINE_LAST_ERROR(linear_attention)
