// The delta rule with a decay per key channel over whole portions of prompts, in chunks of 16 tokens whose rows are computed
// side by side from the state ahead of them.  Per head, with k, q of length d (k, and q before its scale, of unit length),
// g_t the decays and beta_t the step sizes, the recurrence is
//
//   S_t = diag(g_t) S_(t-1) + k_t u_t^T,   u_t = beta_t (v_t - (diag(g_t) S_(t-1))^T k_t),   o_t = S_t^T q_t.
//
// In a chunk that starts from S_0, with b_t the sum of the decays' logarithms up to token t (so that exp(b_t - b_s) <= 1 for
// s <= t: nothing overflows however fast a channel forgets):
//
//   a_ts = sum_c k_t k_s exp(b_t - b_s)  (s < t),   p_ts = sum_c q_t k_s exp(b_t - b_s)  (s <= t)
//   X_t  = beta_t (r_t - sum_(s < t) a_ts X_s),  solved for r_t = k_t exp(b_t) (-> W, [16, d]) and for r_t = v_t (-> Y, [16, dv])
//   U    = Y - W S_0
//   o_t  = (q_t exp(b_t)) S_0 + sum_(s <= t) p_ts u_s
//   S    = diag(exp(b_last)) S_0 + sum_s (k_s exp(b_last - b_s)) u_s^T
//
// delta_chunk_prepare_kernel   all that does not depend on the state, 32-bit on the CUDA cores, a block per chunk and head
// delta_chunk_scan_kernel      the last three lines, a block per head, portion and 16 columns of the state.  The state's
//                              columns are the rows of the tensor-core instruction (m16n8k8, TF32 operands, 32-bit sums), its
//                              channels lie across the warps and stay in accumulators from the first chunk to the last:
//                              as a result of one product they are the left operand of the next without a move (the
//                              instruction's k may run in any order that both operands share).  Every 32-bit operand enters as
//                              two TF32 numbers, hi + lo, and every product as lo hi + hi lo + hi hi, which keeps 21 bits of
//                              the operands: what is left out is of the order of 32-bit rounding.  The next chunk's
//                              numbers arrive by the copy engine, in two runs of bytes, while this one's are used.
//
// What a row is depends on the state and the portion's tokens only.
#include "common.cuh"
#include "tma.cuh"

namespace air {

constexpr int DC = 16;              // tokens of a chunk, and columns of a block of the scan
constexpr int DC_RLD = 40, DC_ULD = 24;      // strides of rows in shared memory: four rows fall into different banks
constexpr float DC_FLOOR = -60.f;   // a decay of 2^-60 is none: the logarithms' sums stay small enough to be exact

// What a chunk and head leave in the scratch memory, DP the channels filled up to 32, 64, 128 or 256 (zeros), in floats:
//   rows [32][DP]     W and q exp b; the eight channels from 8 i on of row t stand at 8 (i ^ (t & 3))
//   keys [DP][16]     (k exp(b_last - b))^T; the eight tokens from 8 i on of channel c stand at 8 (i ^ (c / 2 & 1))
//   last [DP]         exp b_last
//   p    [16][16]     swizzled as the keys are
//   Y^T  [dvp][16]    dvp: dv filled up to a multiple of 16 (zeros)
// (in this arrangement four rows that a warp reads eight bytes at a time fall into different banks)
template <int DP> struct DeltaChunk {
    static constexpr int KEYS = 32 * DP, LAST = KEYS + DC * DP, P = LAST + DP, Y = P + DC * DC;
};
__device__ __forceinline__ int dc_row_place(int t, int c) { return c ^ ((t & 3) << 3); }
__device__ __forceinline__ int dc_key_place(int c, int t) { return t ^ (((c >> 1) & 1) << 3); }

struct DeltaChunkArgs {
    const float* q; int ldq;        // [T, ldq]: head g's d numbers at column g * d, before their unit length and scale
    const float* k; int ldk;
    const float* v; int ldv;        // [T, ldv]: head h's dv numbers at column h * dv
    const float* decay; int ldd;    // [T, ldd]: d logits per head
    const float* beta; int ldb;     // [T, ldb]: one logit per head
    const float* a_log;             // [H]
    const float* dt_bias;           // [H * d]
    const int* chunks;              // [N, 2]: first row, tokens
    const int* portions;            // [L, 4]: first row, tokens, slot, first chunk
    float* scratch;                 // [N, H, stride]
    float* state;                   // [slots, H, d, dv]
    float* out;                     // [T, H, dv]
    int H, G, d, dv, dvp;
    float q_scale, unit_eps;
    long long stride;
    int* status;
};

__device__ __forceinline__ float softplus_1(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// 2^x in one instruction (x <= 0 here; relative error about 2^-22)
__device__ __forceinline__ float power_of_2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int DP>
__global__ void __launch_bounds__(256, DP <= 128 ? 3 : 2) delta_chunk_prepare_kernel(const DeltaChunkArgs p) {
    constexpr int ld = DP + 4, PER = DP / 32;
    extern __shared__ __align__(16) float smem[];
    __shared__ __align__(16) float sa[DC][DC];
    __shared__ float sbeta[DC];
    pdl_enter(TR_SCAN);
    const int h = blockIdx.y, g = h / (p.H / p.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int q0 = p.chunks[2 * blockIdx.x], n = p.chunks[2 * blockIdx.x + 1];
    const int d = p.d;
    float* sk = smem;                       // [16][ld]
    float* sq = sk + DC * ld;
    float* sb = sq + DC * ld;               // the decays' logarithms to the base 2, then their sums
    const float rate = -expf(p.a_log[h]) * 1.4426950408889634f;
    {   // a warp per two tokens: unit lengths, logarithms (both tokens' loads under way at once)
        float x[2][PER], y[2][PER], z[2][PER];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = warp + 8 * r;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int c = lane + 32 * i;
                const bool in = t < n && c < d;
                x[r][i] = in ? p.k[(size_t)(q0 + t) * p.ldk + g * d + c] : 0.f;
                y[r][i] = in ? p.q[(size_t)(q0 + t) * p.ldq + g * d + c] : 0.f;
                z[r][i] = in ? p.decay[(size_t)(q0 + t) * p.ldd + h * d + c] + p.dt_bias[h * d + c] : 0.f;
            }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = warp + 8 * r;
            float ss = 0.f, qs = 0.f;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                ss = fmaf(x[r][i], x[r][i], ss);
                qs = fmaf(y[r][i], y[r][i], qs);
                sb[t * ld + lane + 32 * i] = t < n && lane + 32 * i < d ? fmaxf(rate * softplus_1(z[r][i]), DC_FLOOR) : 0.f;
            }
            const float kf = 1.f / sqrtf(warp_sum(ss) + p.unit_eps), qf = p.q_scale / sqrtf(warp_sum(qs) + p.unit_eps);
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                sk[t * ld + lane + 32 * i] = x[r][i] * kf;
                sq[t * ld + lane + 32 * i] = y[r][i] * qf;
            }
            if (lane == 0) sbeta[t] = t < n ? 1.f / (1.f + expf(-p.beta[(size_t)(q0 + t) * p.ldb + h])) : 0.f;
        }
    }
    __syncthreads();
    if (tid < DP) {
        float sum = 0.f;
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            sum += sb[t * ld + tid];
            sb[t * ld + tid] = sum;
        }
    }
    using Place = DeltaChunk<DP>;
    float* base = p.scratch + ((size_t)blockIdx.x * p.H + h) * p.stride;
    float* Pm = base + Place::P;
    {
        const int t = tid / DC, s = tid % DC;
        if (s > t) {
            sa[t][s] = 0.f;
            Pm[t * DC + dc_key_place(t, s)] = 0.f;
        }
    }
    __syncthreads();
    // a and p: four threads (a quarter of the channels each) per square of 2 x 2 tokens on or below the diagonal, 36 squares
    if (tid < 160) {
        const int square = min(tid >> 2, 35), part = tid & 3;
        int i = 0;
        while ((i + 1) * (i + 2) / 2 <= square) ++i;
        const int j = square - i * (i + 1) / 2;          // tokens 2 i, 2 i + 1 against 2 j, 2 j + 1
        float a[2][2] = {{0.f, 0.f}, {0.f, 0.f}}, pq[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
#pragma unroll 2
        for (int c = part * 4; c < DP; c += 16) {
            float xk[2][4], xq[2][4], xb[2][4], yk[2][4], yb[2][4];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                load4(sk + (2 * i + r) * ld + c, xk[r]);
                load4(sq + (2 * i + r) * ld + c, xq[r]);
                load4(sb + (2 * i + r) * ld + c, xb[r]);
                load4(sk + (2 * j + r) * ld + c, yk[r]);
                load4(sb + (2 * j + r) * ld + c, yb[r]);
            }
#pragma unroll
            for (int r = 0; r < 2; ++r)
#pragma unroll
                for (int s = 0; s < 2; ++s)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        float x = xb[r][e] - yb[s][e];
                        if (r < s) x = fminf(x, 0.f);      // (above the diagonal where i = j: not kept, but it may not overflow)
                        const float w = yk[s][e] * power_of_2(x);
                        a[r][s] = fmaf(xk[r][e], w, a[r][s]);
                        pq[r][s] = fmaf(xq[r][e], w, pq[r][s]);
                    }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int s = 0; s < 2; ++s) {
                a[r][s] += __shfl_xor_sync(0xffffffffu, a[r][s], 1);
                a[r][s] += __shfl_xor_sync(0xffffffffu, a[r][s], 2);
                pq[r][s] += __shfl_xor_sync(0xffffffffu, pq[r][s], 1);
                pq[r][s] += __shfl_xor_sync(0xffffffffu, pq[r][s], 2);
                const int t = 2 * i + r, u = 2 * j + s;
                if (part == 0 && tid < 144 && u <= t) {
                    sa[t][u] = u < t ? sbeta[t] * a[r][s] : 0.f;
                    Pm[t * DC + dc_key_place(t, u)] = pq[r][s];
                }
            }
    }
    __syncthreads();
    // W and Y, a thread per column; what else the scan reads of a channel
    for (int j = tid; j < DP + p.dvp; j += 256) {
        float x[DC];
        if (j < DP) {
            const float last = sb[(DC - 1) * ld + j];
            float* keys = base + Place::KEYS + j * DC;
#pragma unroll
            for (int t = 0; t < DC; t += 4) {
                float kv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float b = sb[(t + i) * ld + j], k = sk[(t + i) * ld + j], e = power_of_2(b);
                    x[t + i] = k * e;
                    base[(DC + t + i) * DP + dc_row_place(t + i, j)] = sq[(t + i) * ld + j] * e;
                    kv[i] = k * power_of_2(last - b);
                }
                store4(keys + dc_key_place(j, t), kv);
            }
            base[Place::LAST + j] = power_of_2(last);
        } else {
            const int c = j - DP;
#pragma unroll
            for (int t = 0; t < DC; ++t) x[t] = t < n && c < p.dv ? p.v[(size_t)(q0 + t) * p.ldv + h * p.dv + c] : 0.f;
        }
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            float sum = sbeta[t] * x[t];
#pragma unroll
            for (int s = 0; s < t; s += 4) {               // (the places on and above the diagonal hold zeros)
                float w[4];
                load4(&sa[t][s], w);
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    if (s + i < t) sum = fmaf(-w[i], x[s + i], sum);
            }
            x[t] = sum;
        }
        if (j < DP) {
#pragma unroll
            for (int t = 0; t < DC; ++t) base[t * DP + dc_row_place(t, j)] = x[t];
        } else {
            float* dst = base + Place::Y + (j - DP) * DC;
#pragma unroll
            for (int t = 0; t < DC; t += 4) {
                const float y[4] = {x[t], x[t + 1], x[t + 2], x[t + 3]};
                store4(dst + t, y);
            }
        }
    }
}

// A 32-bit number as two TF32 numbers: the instruction reads the upper 19 bits of an operand.
struct Two { uint32_t hi, lo; };
__device__ __forceinline__ Two two_of(float x) {
    const uint32_t hi = __float_as_uint(x) & 0xffffe000u;
    return Two{hi, __float_as_uint(x - __uint_as_float(hi))};
}
// c += a b; with k in the order that the accumulators have: a holds (row g, k 2t), (g + 8, 2t), (g, 2t + 1), (g + 8, 2t + 1), b
// holds (k 2t, column g), (2t + 1, g)
__device__ __forceinline__ void mma_tf32(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
                 "{%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void two_pair(Two (&b)[2], const float* p) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    b[0] = two_of(v.x);
    b[1] = two_of(v.y);
}

constexpr int DC_WARPS = 4;         // one per scheduler: the products follow one another in the tensor pipe as fast as it takes them,
                                    // and the fewer warps share the channels, the fewer sums cross between them
constexpr int DC_STAGES = 2;

// A warp holds NJ tiles of 8 channels of the state, transposed: S[j] is (column g or g + 8 of the block) x (channels 8 j + 2 t,
// 8 j + 2 t + 1), g = lane / 4, t = lane % 4.
template <int DP>
__global__ void __launch_bounds__(DC_WARPS * 32) delta_chunk_scan_kernel(const DeltaChunkArgs p) {
    constexpr int NJ = DP / (8 * DC_WARPS);
    constexpr int STAGES = DC_STAGES, BUF = DeltaChunk<DP>::Y + DC * DC;      // floats of a buffer: the chunk's, and 16 columns of Y
    using Place = DeltaChunk<DP>;
    extern __shared__ __align__(16) float smem[];
    __shared__ __align__(8) uint64_t full[STAGES];
    __shared__ int gave_up;
    float* red = smem + STAGES * BUF;       // [warps][16 columns][DC_RLD]: 32 sums over a warp's channels
    float* UT = red + DC_WARPS * DC * DC_RLD;   // [16 columns][DC_ULD]: U transposed
    float* OT = UT + DC * DC_ULD;           // the same of o's first part
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t2 = 2 * (lane & 3);
    if (tid == 0) {
        for (int i = 0; i < STAGES; ++i) mbar_init(&full[i], 1);
        gave_up = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_enter(TR_SCAN);
    const int h = blockIdx.y, col0 = blockIdx.x * DC;
    const int* por = p.portions + 4 * blockIdx.z;
    const int row0 = por[0], tokens = por[1], slot = por[2], chunk0 = por[3];
    if (slot < 0) return;
    const int chunks = (tokens + DC - 1) / DC;
    auto stage = [&](int i) {               // (one thread)
        const float* src = p.scratch + ((size_t)(chunk0 + i) * p.H + h) * p.stride;
        float* dst = smem + (i % STAGES) * BUF;
        uint64_t* bar = &full[i % STAGES];
        mbar_expect_tx(bar, BUF * 4);
        bulk_load(dst, src, Place::Y * 4, bar);
        bulk_load(dst + Place::Y, src + Place::Y + col0 * DC, DC * DC * 4, bar);
    };
    if (tid == 0)
        for (int i = 0; i < min(STAGES - 1, chunks); ++i) stage(i);
    const int r0 = warp * 8 * NJ;
    float* st = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
    float S[NJ][4];
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = r0 + 8 * j + t2 + (e & 1), c = col0 + g + 8 * (e >> 1);
            S[j][e] = r < p.d && c < p.dv ? st[(size_t)r * p.dv + c] : 0.f;
        }
    // places that do not change from chunk to chunk
    const int rows_at = g * DP + t2, swap = dc_key_place(g, 0);      // (of rows 8 j + g: the tile does not matter)
    float* mine = red + (warp * DC + g) * DC_RLD + t2;
    const int sum_c = tid >> 3, sum_t = 4 * (tid & 7);               // the four sums that this thread completes: column, rows
    const float* sum_from = red + sum_c * DC_RLD + sum_t;
    float* sum_to = (sum_t < DC ? UT : OT - DC) + sum_c * DC_ULD + sum_t;
    const int t0 = 8 * (warp & 1);                                   // warps 0 and 1: the tokens whose o they finish
    float* out = p.out + ((size_t)(row0 + t0 + t2) * p.H + h) * p.dv + col0 + g;
    const size_t out_row = (size_t)p.H * p.dv;
    for (int i = 0; i < chunks; ++i) {
        const float* buf = smem + (i % STAGES) * BUF;
        const bool ok = mbar_wait(&full[i % STAGES], (i / STAGES) & 1, &gave_up);
        // this chunk's numbers are there and everybody is done with the chunk before it
        if (__syncthreads_or(!ok)) {
            for (int x = 0; x < 32; ++x) __nanosleep(2000);      // (a copy on its way may still land)
            if (tid == 0 && p.status) atomicExch(p.status, 9);
            return;
        }
        if (tid == 0 && i + STAGES - 1 < chunks) stage(i + STAGES - 1);
        float acc[4][4];
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[x][0] = acc[x][1] = acc[x][2] = acc[x][3] = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const Two a[4] = {two_of(S[j][0]), two_of(S[j][2]), two_of(S[j][1]), two_of(S[j][3])};
            const float* at = buf + rows_at + dc_row_place(g, r0 + 8 * j);
            Two b[4][2];
#pragma unroll
            for (int x = 0; x < 4; ++x) two_pair(b[x], at + 8 * x * DP);
            // (the four sums in turn: a product does not wait for the one before it)
#pragma unroll
            for (int x = 0; x < 4; ++x) mma_tf32(acc[x], a[0].lo, a[1].lo, a[2].lo, a[3].lo, b[x][0].hi, b[x][1].hi);
#pragma unroll
            for (int x = 0; x < 4; ++x) mma_tf32(acc[x], a[0].hi, a[1].hi, a[2].hi, a[3].hi, b[x][0].lo, b[x][1].lo);
#pragma unroll
            for (int x = 0; x < 4; ++x) mma_tf32(acc[x], a[0].hi, a[1].hi, a[2].hi, a[3].hi, b[x][0].hi, b[x][1].hi);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            *reinterpret_cast<float2*>(mine + 8 * x) = make_float2(acc[x][0], acc[x][1]);
            *reinterpret_cast<float2*>(mine + 8 * DC_RLD + 8 * x) = make_float2(acc[x][2], acc[x][3]);
        }
        __syncthreads();
        {   // the warps' sums in order: U = Y - W S (rows 0 .. 15 of 32), o's first part (the others)
            float v[DC_WARPS][4];
#pragma unroll
            for (int w = 0; w < DC_WARPS; ++w) load4(sum_from + w * DC * DC_RLD, v[w]);
            float y[4] = {0.f, 0.f, 0.f, 0.f};
            if (sum_t < DC) load4(buf + Place::Y + sum_c * DC + sum_t, y);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float sum = (v[0][e] + v[1][e]) + (v[2][e] + v[3][e]);
                y[e] = sum_t < DC ? y[e] - sum : sum;
            }
            store4(sum_to, y);
        }
        __syncthreads();
        Two u[2][4];                         // U transposed, tokens 0 .. 7 and 8 .. 15
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            Two lo[2], hi[2];
            two_pair(lo, UT + g * DC_ULD + 8 * x + t2);
            two_pair(hi, UT + (g + 8) * DC_ULD + 8 * x + t2);
            u[x][0] = lo[0]; u[x][1] = hi[0]; u[x][2] = lo[1]; u[x][3] = hi[1];
        }
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const float2 e = *reinterpret_cast<const float2*>(buf + Place::LAST + r0 + 8 * j + t2);
            S[j][0] *= e.x; S[j][1] *= e.y; S[j][2] *= e.x; S[j][3] *= e.y;
        }
        float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            Two k[NJ][2], w[2];
#pragma unroll
            for (int j = 0; j < NJ; ++j)
                two_pair(k[j], buf + Place::KEYS + (r0 + 8 * j + g) * DC + ((8 * x) ^ swap) + t2);
            if (warp < 2) {                  // o: its products stand among the state's, which do not wait for them
                if (x == 0) {
                    const float2 lo = *reinterpret_cast<const float2*>(OT + g * DC_ULD + t0 + t2);
                    const float2 hi = *reinterpret_cast<const float2*>(OT + (g + 8) * DC_ULD + t0 + t2);
                    o[0] = lo.x; o[1] = lo.y; o[2] = hi.x; o[3] = hi.y;
                }
                two_pair(w, buf + Place::P + (t0 + g) * DC + ((8 * x) ^ swap) + t2);
                mma_tf32(o, u[x][0].lo, u[x][1].lo, u[x][2].lo, u[x][3].lo, w[0].hi, w[1].hi);
            }
#pragma unroll
            for (int j = 0; j < NJ; ++j) mma_tf32(S[j], u[x][0].lo, u[x][1].lo, u[x][2].lo, u[x][3].lo, k[j][0].hi, k[j][1].hi);
            if (warp < 2) mma_tf32(o, u[x][0].hi, u[x][1].hi, u[x][2].hi, u[x][3].hi, w[0].lo, w[1].lo);
#pragma unroll
            for (int j = 0; j < NJ; ++j) mma_tf32(S[j], u[x][0].hi, u[x][1].hi, u[x][2].hi, u[x][3].hi, k[j][0].lo, k[j][1].lo);
            if (warp < 2) mma_tf32(o, u[x][0].hi, u[x][1].hi, u[x][2].hi, u[x][3].hi, w[0].hi, w[1].hi);
#pragma unroll
            for (int j = 0; j < NJ; ++j) mma_tf32(S[j], u[x][0].hi, u[x][1].hi, u[x][2].hi, u[x][3].hi, k[j][0].hi, k[j][1].hi);
        }
        if (warp < 2) {
            float* to = out + (size_t)i * DC * out_row;
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (i * DC + t0 + t2 + (e & 1) < tokens && col0 + g + 8 * (e >> 1) < p.dv)
                    to[(e & 1) * out_row + 8 * (e >> 1)] = o[e];
        }
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = r0 + 8 * j + t2 + (e & 1), c = col0 + g + 8 * (e >> 1);
            if (r < p.d && c < p.dv) st[(size_t)r * p.dv + c] = S[j][e];
        }
}

template <int DP>
static int launch_delta_chunks(const DeltaChunkArgs& args, int N, int L, cudaStream_t stream) {
    DeltaChunkArgs a = args;
    a.dvp = (a.dv + 15) / 16 * 16;
    a.stride = DeltaChunk<DP>::Y + (long long)DC * a.dvp;
    const size_t smem1 = sizeof(float) * 3 * DC * (DP + 4);
    if (smem1 > 44 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
        if (e != cudaSuccess) return (int)e;
    }
    int rc = launch(delta_chunk_prepare_kernel<DP>, dim3(N, a.H), 256, smem1, stream, a);
    if (rc) return rc;
    size_t smem2 = sizeof(float) * (DC_STAGES * (DeltaChunk<DP>::Y + DC * DC) + DC_WARPS * DC * DC_RLD + 2 * DC * DC_ULD);
    const dim3 grid(a.dvp / DC, a.H, L);
    // (as for the scan token by token: the blocks start when their predecessor has ended, and spread over the SMs)
    int sms = 148, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long blocks = (long long)grid.x * grid.y * grid.z;
    if (blocks <= sms && smem2 < 120 * 1024) smem2 = 120 * 1024;
    cudaError_t e = cudaFuncSetAttribute(delta_chunk_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem2);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(DC_WARPS * 32);
    cfg.dynamicSmemBytes = smem2;
    cfg.stream = stream;
    return (int)cudaLaunchKernelEx(&cfg, delta_chunk_scan_kernel<DP>, a);
}

}  // namespace air

// scratch: float32 [N, H, 49 DP + 256 + 16 dvp] with DP = d filled up to 32, 64, 128 or 256, dvp = dv to a multiple of 16.
// Rows and slots as the lists say; d up to 256.
AIR_API int air_delta_portions(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* decay,
                               int ldd, const float* beta, int ldb, const float* a_log, const float* dt_bias, float* state,
                               float* out, const int* portions, int L, const int* chunks, int N, float* scratch, int H, int G,
                               int d, int dv, float q_scale, float unit_eps, int* status, cudaStream_t stream) {
    using namespace air;
    if (L <= 0 || N <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || d > 256 || dv <= 0 || H > 65535 || L > 65535 || !scratch ||
        ((uintptr_t)scratch & 15))
        return AIR_ERR_BAD_ARGUMENT;
    DeltaChunkArgs a;
    a.q = q; a.ldq = ldq; a.k = k; a.ldk = ldk; a.v = v; a.ldv = ldv; a.decay = decay; a.ldd = ldd; a.beta = beta; a.ldb = ldb;
    a.a_log = a_log; a.dt_bias = dt_bias; a.chunks = chunks; a.portions = portions; a.scratch = scratch; a.state = state;
    a.out = out; a.H = H; a.G = G; a.d = d; a.dv = dv; a.dvp = 0; a.q_scale = q_scale; a.unit_eps = unit_eps; a.stride = 0;
    a.status = status;
    if (d <= 32) return launch_delta_chunks<32>(a, N, L, stream);
    if (d <= 64) return launch_delta_chunks<64>(a, N, L, stream);
    if (d <= 128) return launch_delta_chunks<128>(a, N, L, stream);
    return launch_delta_chunks<256>(a, N, L, stream);
}

AIR_API int air_trace_set_delta_chunks(unsigned long long* buffer) { return air::set_trace_here(buffer); }
