// Row-wise operations of layers that carry several residual streams side by side (hyper-connections), of layer norms with
// a bias, and of a convolution over time that is added to its own input.
//
//   stream_norm_kernel    with the streams x_0 .. x_(S-1) [T, E] (S = 1: an ordinary residual stream) and the output y of
//                         the sub-layer before (float32 [T, E], or the partial sums [parts, T, E] of a split product, added
//                         in order):
//                           x'_t = sum_s mix[s, t] x_s + out_t y     (without mix: x_t; without out: y as it is)
//                           u    = sum_t read_t x'_t                 (without read: the plain sum)
//                           row  = norm(u) * w + b
//                         where norm is (u - mean) / sqrt(var + eps), var the mean of the squared deviations, or (center 0)
//                         u / sqrt(mean(u^2) + eps), and b may be absent.  x' is written when h_out is given; with `rows` the
//                         kernel reads row rows[r] of everything and writes row r.  The streams may all be one tensor
//                         (stream stride 0: they start out equal).  Everything is 32-bit; the row is written in its own type.
//                         More terms than y may join the one stream of an ordinary layer (S = 1) in the same pass: up to
//                         two, each a tensor or partial sums, each with a factor per row (the sub-layers of a layer that
//                         stand side by side, one of them with a gate per token).  Without w but with `out` the row
//                         is written as it is, no norm, ahead of the row of a second tensor where one is given: [u | again],
//                         2 E columns.
//                         With conv (a step in which every row is its request's only token) the row becomes
//                         row + sum_j cw[j] in_(t - taps + 1 + j) before it is written, the earlier inputs coming from
//                         the request's state, which is moved on by one token.
//   residual_conv_kernel  y_t = h_t + sum_j cw[j] h_(t - taps + 1 + j) over the tokens of each entry of the batch: the same
//                         convolution for portions of any length.
//
// cw is [taps, E] (the last row multiplies the token itself), the state [slots, taps - 1, E], oldest input first, zeros at
// a request's start.
#include "common.cuh"

namespace air {

// One more term of the sum into an ordinary residual stream: partial sums [parts, T, E], times a factor per row (or 1).
struct StreamTerm {
    const float* y; int parts; const float* gate;
};
constexpr int STREAM_MORE = 2;

struct StreamNormArgs {
    const float* x; size_t x_stride;       // stream s at x + s * x_stride
    float* h_out; size_t h_stride;         // may be x itself (a thread reads its columns of all streams before it writes)
    const float* y; int y_parts; size_t part_stride;
    const float* mix;                      // [S, S], from row s to column t
    const float* out_w;                    // [S]
    const float* read;                     // [S]
    const float* w; const float* b;        // [E]
    void* out;
    const int* rows;
    const float* conv_w; float* conv_state; const int* token_seq; int taps;
    int S, E, center;
    float eps;
    StreamTerm more[STREAM_MORE];          // (S = 1)
    const float* again;                    // [T, E], written behind the row where there is no norm
};

constexpr int STREAMS_MAX = 16;

template <int N> __device__ __forceinline__ void load_columns(const float* q, float (&v)[N]) {
    if constexpr (N == 4) load4(q, v);
    else v[0] = *q;
}
template <int N> __device__ __forceinline__ void store_columns(float* q, const float (&v)[N]) {
    if constexpr (N == 4) store4(q, v);
    else *q = v[0];
}

// N columns of all streams of a row: mixed, written, and folded into u.  NS: the number of streams, all at compile-time
// indices; 0: p.S of them, in a loop.
template <int NS, int N>
__device__ __forceinline__ void stream_columns(const StreamNormArgs& p, int row, int i, const float* coef, float (&u)[N]) {
    const size_t src = (size_t)row * p.E;
    const int S = NS ? NS : p.S;
    constexpr int UN = NS ? NS : 1;
    float x[NS ? NS : STREAMS_MAX][N], y[N];
#pragma unroll UN
    for (int s = 0; s < S; ++s) load_columns<N>(p.x + s * p.x_stride + src + i, x[s]);
    if (p.y) {
        load_columns<N>(p.y + src + i, y);
#pragma unroll 4
        for (int q = 1; q < p.y_parts; ++q) {                                        // (loads ahead, sums in order)
            float t[N];
            load_columns<N>(p.y + q * p.part_stride + src + i, t);
#pragma unroll
            for (int j = 0; j < N; ++j) y[j] += t[j];
        }
        if constexpr (NS <= 1) {
#pragma unroll
            for (int m = 0; m < STREAM_MORE; ++m) {
                const StreamTerm& term = p.more[m];
                if (!term.y) continue;
                float z[N];
                load_columns<N>(term.y + src + i, z);
#pragma unroll 4
                for (int q = 1; q < term.parts; ++q) {
                    float t[N];
                    load_columns<N>(term.y + q * p.part_stride + src + i, t);
#pragma unroll
                    for (int j = 0; j < N; ++j) z[j] += t[j];
                }
                const float g = term.gate ? term.gate[row] : 1.f;
#pragma unroll
                for (int j = 0; j < N; ++j) y[j] = fmaf(g, z[j], y[j]);
            }
        }
    }
    const float *mix = coef, *out_w = coef + S * S, *read = out_w + S;
#pragma unroll
    for (int j = 0; j < N; ++j) u[j] = 0.f;
#pragma unroll UN
    for (int t = 0; t < S; ++t) {
        float v[N];
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = p.mix ? 0.f : x[t][j];
        if (p.mix)
#pragma unroll UN
            for (int s = 0; s < S; ++s)
#pragma unroll
                for (int j = 0; j < N; ++j) v[j] = fmaf(mix[s * S + t], x[s][j], v[j]);
        if (p.y)
#pragma unroll
            for (int j = 0; j < N; ++j) v[j] = fmaf(out_w[t], y[j], v[j]);
        if (p.h_out) store_columns<N>(p.h_out + t * p.h_stride + src + i, v);
#pragma unroll
        for (int j = 0; j < N; ++j) u[j] = fmaf(read[t], v[j], u[j]);
    }
}

// The finished row's columns i .. i + N - 1: weight and bias, the convolution (slot >= 0), the write.
template <typename TO, int N>
__device__ __forceinline__ void stream_finish(const StreamNormArgs& p, TO* out, int slot, int i, const float (&u)[N], float mean,
                                              float scale, const float (&wv)[N], const float (&bv)[N]) {
    float v[N];
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = (u[j] - mean) * scale * wv[j] + bv[j];
    if (slot >= 0) {      // (four earlier inputs and their weights under way at a time)
        const int keep = p.taps - 1, E = p.E;
        float* st = p.conv_state + (size_t)slot * keep * E + i;
        const float* cw = p.conv_w + i;
        float acc[N];
        load_columns<N>(cw + (size_t)keep * E, acc);
#pragma unroll
        for (int j = 0; j < N; ++j) acc[j] = fmaf(acc[j], v[j], v[j]);
        for (int k0 = 0; k0 < keep; k0 += 4) {
            float in[4][N], wk[4][N];
#pragma unroll
            for (int u2 = 0; u2 < 4; ++u2)
                if (k0 + u2 < keep) {
                    load_columns<N>(st + (size_t)(k0 + u2) * E, in[u2]);
                    load_columns<N>(cw + (size_t)(k0 + u2) * E, wk[u2]);
                }
#pragma unroll
            for (int u2 = 0; u2 < 4; ++u2)
                if (k0 + u2 < keep) {
#pragma unroll
                    for (int j = 0; j < N; ++j) acc[j] = fmaf(wk[u2][j], in[u2][j], acc[j]);
                    if (k0 + u2 > 0) store_columns<N>(st + (size_t)(k0 + u2 - 1) * E, in[u2]);
                }
        }
        if (keep > 0) store_columns<N>(st + (size_t)(keep - 1) * E, v);
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = acc[j];
    }
    if constexpr (N == 4) store4(out + i, v);
    else out[i] = from_float<TO>(v[0]);
}

// A block per row.  ONE: a thread has one piece of N columns at most (few rows: a decode step), which stays in registers, and
// has its weights before the predecessor's rows are there; else the row waits in shared memory between the passes.
template <typename TO, int NS, int N, bool ONE>
__global__ void __launch_bounds__(1024) stream_norm_kernel(const StreamNormArgs p) {
    __shared__ float scratch[32];
    __shared__ float coef[STREAMS_MAX * STREAMS_MAX + 2 * STREAMS_MAX];
    extern __shared__ __align__(16) float urow[];
    const int E = p.E, S = NS ? NS : p.S, first = threadIdx.x * N;
    pdl_trigger();
    // what no kernel writes
    for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {
        const int k = i - S * S;
        coef[i] = k < 0 ? (p.mix ? p.mix[i] : 0.f) : k < S ? (p.out_w ? p.out_w[k] : 1.f) : (p.read ? p.read[k - S] : 1.f);
    }
    float w1[N], b1[N];
#pragma unroll
    for (int j = 0; j < N; ++j) w1[j] = b1[j] = 0.f;
    if (ONE && p.w && first < E) {
        load_columns<N>(p.w + first, w1);
        if (p.b) load_columns<N>(p.b + first, b1);
    }
    __syncthreads();
    pdl_wait();
    trace_point(TR_STREAM_NORM);
    const int r = blockIdx.x;
    const int row = p.rows ? p.rows[r] : r;
    const size_t src = (size_t)row * E;
    const int step = blockDim.x * N;
    float u1[N], sum = 0.f;
#pragma unroll
    for (int j = 0; j < N; ++j) u1[j] = 0.f;
    if constexpr (ONE) {
        if (first < E) stream_columns<NS, N>(p, row, first, coef, u1);
#pragma unroll
        for (int j = 0; j < N; ++j) sum += p.center ? u1[j] : u1[j] * u1[j];
    } else {
        for (int i = first; i < E; i += step) {
            float u[N];
            stream_columns<NS, N>(p, row, i, coef, u);
#pragma unroll
            for (int j = 0; j < N; ++j) {
                urow[i + j] = u[j];
                sum += p.center ? u[j] : u[j] * u[j];
            }
        }
    }
    if (!p.w) {
        if (!p.out) return;
        // the row as it is, and the second tensor's row behind it
        const int width = p.again ? 2 * E : E;
        TO* out = (TO*)p.out + (size_t)r * width;
        for (int i = first; i < E; i += step) {
            float u[N], a[N];
#pragma unroll
            for (int j = 0; j < N; ++j) u[j] = ONE ? u1[j] : urow[i + j];
            if constexpr (N == 4) store4(out + i, u);
            else out[i] = from_float<TO>(u[0]);
            if (!p.again) continue;
            load_columns<N>(p.again + src + i, a);
            if constexpr (N == 4) store4(out + E + i, a);
            else out[E + i] = from_float<TO>(a[0]);
        }
        return;
    }
    float mean = 0.f;
    if (p.center) {
        mean = block_sum(sum, scratch) / (float)E;
        sum = 0.f;
        if constexpr (ONE) {
#pragma unroll
            for (int j = 0; j < N; ++j) {
                const float d = u1[j] - mean;
                if (first < E) sum = fmaf(d, d, sum);
            }
        } else {
            for (int i = first; i < E; i += step)
#pragma unroll
                for (int j = 0; j < N; ++j) {
                    const float d = urow[i + j] - mean;
                    sum = fmaf(d, d, sum);
                }
        }
    }
    const float scale = 1.f / sqrtf(block_sum(sum, scratch) / (float)E + p.eps);
    TO* out = (TO*)p.out + (size_t)r * E;
    const int slot = p.conv_w ? p.token_seq[r] : -1;
    if constexpr (ONE) {
        if (first < E) stream_finish<TO, N>(p, out, slot, first, u1, mean, scale, w1, b1);
    } else {
        for (int i = first; i < E; i += step) {
            float u[N], wv[N], bv[N];
#pragma unroll
            for (int j = 0; j < N; ++j) {
                u[j] = urow[i + j];
                bv[j] = 0.f;
            }
            load_columns<N>(p.w + i, wv);
            if (p.b) load_columns<N>(p.b + i, bv);
            stream_finish<TO, N>(p, out, slot, i, u, mean, scale, wv, bv);
        }
    }
}

// grid (column blocks, entries, chunks of `chunk` tokens, at least taps - 1); a thread takes N columns.  The thread of a
// column in an entry's first chunk is the only one that reads or writes that column's state.
template <typename TO, int N>
__global__ void __launch_bounds__(128)
residual_conv_kernel(const float* __restrict__ h, const float* __restrict__ w, float* __restrict__ state,
                     TO* __restrict__ y, const int* __restrict__ q_start, const int* __restrict__ slots, int E, int taps,
                     int chunk) {
    pdl_enter(TR_RESIDUAL_CONV);
    const int i = (blockIdx.x * 128 + threadIdx.x) * N, e = blockIdx.y;
    const int slot = slots[e];
    if (i >= E || slot < 0) return;
    const int q0 = q_start[e], n = q_start[e + 1] - q0, keep = taps - 1;
    const int t0 = blockIdx.z * chunk, t1 = min(n, t0 + chunk);
    if (t0 >= n) return;
    auto ld = [](const float* q, float (&v)[N]) {
        if constexpr (N == 4) load4(q, v);
        else v[0] = *q;
    };
    const float* in = h + (size_t)q0 * E + i;
    float* st = state + (size_t)slot * keep * E + i;
    for (int t = t0; t < t1; ++t) {
        float cur[N], acc[N], v[N], wv[N];
        ld(in + (size_t)t * E, cur);
        ld(w + (size_t)keep * E + i, wv);
#pragma unroll
        for (int j = 0; j < N; ++j) acc[j] = fmaf(wv[j], cur[j], cur[j]);
        for (int k = 0; k < keep; ++k) {
            const int back = t - keep + k;
            ld(back >= 0 ? in + (size_t)back * E : st + (size_t)(keep + back) * E, v);
            ld(w + (size_t)k * E + i, wv);
#pragma unroll
            for (int j = 0; j < N; ++j) acc[j] = fmaf(wv[j], v[j], acc[j]);
        }
        if constexpr (N == 4) store4(y + (size_t)(q0 + t) * E + i, acc);
        else y[(size_t)(q0 + t) * E + i] = from_float<TO>(acc[0]);
    }
    if (blockIdx.z == 0)
        for (int k = 0; k < keep; ++k) {       // the entry's last taps - 1 inputs (older ones were in the state already)
            float v[N];
            const int at = n - keep + k;
            ld(at >= 0 ? in + (size_t)at * E : st + (size_t)(keep + at) * E, v);
            if constexpr (N == 4) store4(st + (size_t)k * E, v);
            else st[(size_t)k * E] = v[0];
        }
}

}  // namespace air

AIR_API int air_stream_norm(const float* x, long long x_stride, float* h_out, long long h_stride, const float* y, int y_parts,
                            long long part_stride, const float* mix, const float* out_w, const float* read, int S,
                            const float* w, const float* b, void* out, int out_dtype, const int* rows, int R, int E,
                            int center, float eps, const float* conv_w, float* conv_state, const int* token_seq, int taps,
                            const float* more1, int more1_parts, const float* gate1, const float* more2, int more2_parts,
                            const float* gate2, const float* again, cudaStream_t stream) {
    if (R <= 0) return 0;
    if ((more1 || more2) && (S != 1 || !y || (more1 && more1_parts < 1) || (more2 && more2_parts < 1)))
        return AIR_ERR_BAD_ARGUMENT;
    if (again && (w || !out)) return AIR_ERR_BAD_ARGUMENT;
    if (!x || S < 1 || S > air::STREAMS_MAX || E <= 0 || (y && y_parts < 1) || (w && !out) || (conv_w && (taps < 1 || rows || !token_seq)) ||
        (conv_w && taps > 1 && !conv_state))
        return AIR_ERR_BAD_ARGUMENT;
    const size_t smem = sizeof(float) * (size_t)E;
    if (smem > 200 * 1024) return AIR_ERR_BAD_ARGUMENT;
    air::StreamNormArgs p;
    p.x = x; p.x_stride = (size_t)x_stride; p.h_out = h_out; p.h_stride = (size_t)h_stride; p.y = y; p.y_parts = y_parts;
    p.part_stride = (size_t)part_stride; p.mix = mix; p.out_w = out_w; p.read = read; p.S = S; p.w = w; p.b = b; p.out = out;
    p.rows = rows; p.E = E; p.center = center; p.eps = eps; p.conv_w = conv_w; p.conv_state = conv_state;
    p.token_seq = token_seq; p.taps = taps;
    p.more[0] = air::StreamTerm{more1, more1_parts, gate1}; p.more[1] = air::StreamTerm{more2, more2_parts, gate2};
    p.again = again;
    auto al = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
    const bool vec = E % 4 == 0 && x_stride % 4 == 0 && h_stride % 4 == 0 && part_stride % 4 == 0 && al(x) && al(h_out) &&
                     al(y) && al(w) && al(b) && al(out) && al(conv_w) && al(conv_state) && al(more1) && al(more2) && al(again);
    // few rows: one access of a thread per row, all of a row's loads under way at once
    const int items = vec && S <= 4 ? E / 4 : E;
    int threads = items >= 256 ? 256 : (items + 31) / 32 * 32;
    if (R <= 256) threads = items >= 1024 ? 1024 : (items + 31) / 32 * 32;
    AIR_DISPATCH(out_dtype, TO, {
        auto go = [&](auto kernel, size_t row) {
            if (row > 44 * 1024) {
                cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)row);
                if (err != cudaSuccess) return (int)err;
            }
            return air::launch(kernel, R, threads, row, stream, p);
        };
        const bool one = items <= threads;
        if (!vec || S > 4)
            return one ? go(air::stream_norm_kernel<TO, 0, 1, true>, 0) : go(air::stream_norm_kernel<TO, 0, 1, false>, smem);
        switch (S) {
            case 1: return one ? go(air::stream_norm_kernel<TO, 1, 4, true>, 0) : go(air::stream_norm_kernel<TO, 1, 4, false>, smem);
            case 2: return one ? go(air::stream_norm_kernel<TO, 2, 4, true>, 0) : go(air::stream_norm_kernel<TO, 2, 4, false>, smem);
            case 3: return one ? go(air::stream_norm_kernel<TO, 3, 4, true>, 0) : go(air::stream_norm_kernel<TO, 3, 4, false>, smem);
            default: return one ? go(air::stream_norm_kernel<TO, 4, 4, true>, 0) : go(air::stream_norm_kernel<TO, 4, 4, false>, smem);
        }
    });
    return 0;
}

AIR_API int air_residual_conv(const float* h, const float* w, float* state, void* y, int out_dtype, const int* q_start,
                              const int* slots, int entries, int E, int taps, int max_tokens, cudaStream_t stream) {
    if (entries <= 0 || E <= 0) return 0;
    if (taps < 1 || (taps > 1 && !state) || entries > 65535) return AIR_ERR_BAD_ARGUMENT;
    const int chunk = taps - 1 > 16 ? taps - 1 : 16;
    const int chunks = (max_tokens + chunk - 1) / chunk < 1 ? 1 : (max_tokens + chunk - 1) / chunk;
    if (chunks > 65535) return AIR_ERR_BAD_ARGUMENT;
    const bool vec = E % 4 == 0 && (((uintptr_t)h | (uintptr_t)w | (uintptr_t)state | (uintptr_t)y) & 15) == 0;
    const int items = vec ? E / 4 : E;
    const dim3 grid((items + 127) / 128, entries, chunks);
    AIR_DISPATCH(out_dtype, TO, {
        if (vec)
            return air::launch(air::residual_conv_kernel<TO, 4>, grid, 128, 0, stream, h, w, state, (TO*)y, q_start, slots,
                               E, taps, chunk);
        return air::launch(air::residual_conv_kernel<TO, 1>, grid, 128, 0, stream, h, w, state, (TO*)y, q_start, slots, E,
                           taps, chunk);
    });
    return 0;
}

AIR_API int air_trace_set_stream_ops(unsigned long long* buffer) { return air::set_trace_here(buffer); }
