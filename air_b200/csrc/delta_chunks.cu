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
//                              two TF32 numbers, hi + lo, and every product as lo hi + hi lo + hi hi, which keeps 22 bits of
//                              the operands: what is left out is of the order of 32-bit rounding.  The next chunk's
//                              numbers arrive (cp.async) while this one's are used.
//
// What a row is depends on the state and the portion's tokens only.
#include "common.cuh"

namespace air {

constexpr int DC = 16;              // tokens of a chunk, and columns of a block of the scan
constexpr int DC_MAX_D = 256;
constexpr int DC_KLD = 24, DC_RLD = 40, DC_ULD = 24;      // staged rows' strides: four rows fall into different banks
constexpr float DC_FLOOR = -60.f;   // a decay of 2^-60 is none: the logarithms' sums stay small enough to be exact

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
    int H, G, d, dv, dp, dvp;       // dp: d filled up to a multiple of 16, dvp: dv to one of 4
    float q_scale, unit_eps;
    long long stride;               // of a chunk and head: W, q exp b [16, dp] each, (k exp(b_last - b))^T [dp, 16],
                                    // exp b_last [dp], p [16, 16], Y [16, dvp]
};

__device__ __forceinline__ float softplus_1(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// 2^x in one instruction (x <= 0 here; relative error about 2^-22)
__device__ __forceinline__ float power_of_2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__global__ void __launch_bounds__(256, 2) delta_chunk_prepare_kernel(const DeltaChunkArgs p) {
    extern __shared__ __align__(16) float smem[];
    __shared__ __align__(16) float sa[DC][DC];
    __shared__ float sbeta[DC];
    pdl_enter(TR_SCAN);
    const int h = blockIdx.y, g = h / (p.H / p.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int q0 = p.chunks[2 * blockIdx.x], n = p.chunks[2 * blockIdx.x + 1];
    const int d = p.d, dp = p.dp, ld = dp + 4;
    float* sk = smem;                       // [16][ld]
    float* sq = sk + DC * ld;
    float* sb = sq + DC * ld;               // the decays' logarithms to the base 2, then their sums
    const float rate = -expf(p.a_log[h]) * 1.4426950408889634f;
    for (int t = warp; t < DC; t += 8) {    // a warp per token: unit lengths, logarithms
        const float* kin = p.k + (size_t)(q0 + t) * p.ldk + g * d;
        const float* qin = p.q + (size_t)(q0 + t) * p.ldq + g * d;
        const float* zin = p.decay + (size_t)(q0 + t) * p.ldd + h * d;
        float x[DC_MAX_D / 32], y[DC_MAX_D / 32], ss = 0.f, qs = 0.f;
#pragma unroll
        for (int i = 0; i < DC_MAX_D / 32; ++i) {
            const int c = lane + 32 * i;
            const bool in = t < n && c < d;
            x[i] = in ? kin[c] : 0.f;
            y[i] = in ? qin[c] : 0.f;
            ss = fmaf(x[i], x[i], ss);
            qs = fmaf(y[i], y[i], qs);
            if (c < dp) sb[t * ld + c] = in ? fmaxf(rate * softplus_1(zin[c] + p.dt_bias[h * d + c]), DC_FLOOR) : 0.f;
        }
        const float kf = 1.f / sqrtf(warp_sum(ss) + p.unit_eps), qf = p.q_scale / sqrtf(warp_sum(qs) + p.unit_eps);
#pragma unroll
        for (int i = 0; i < DC_MAX_D / 32; ++i) {
            const int c = lane + 32 * i;
            if (c < dp) {
                sk[t * ld + c] = x[i] * kf;
                sq[t * ld + c] = y[i] * qf;
            }
        }
        if (lane == 0) sbeta[t] = t < n ? 1.f / (1.f + expf(-p.beta[(size_t)(q0 + t) * p.ldb + h])) : 0.f;
    }
    __syncthreads();
    for (int c = tid; c < dp; c += 256) {
        float sum = 0.f;
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            sum += sb[t * ld + c];
            sb[t * ld + c] = sum;
        }
    }
    float* base = p.scratch + ((size_t)blockIdx.x * p.H + h) * p.stride;
    float* W = base;
    float* Qe = W + (size_t)dp * DC;
    float* Kt = Qe + (size_t)dp * DC;
    float* E = Kt + (size_t)DC * dp;
    float* Pm = E + dp;
    float* Y = Pm + DC * DC;
    {
        const int t = tid / DC, s = tid % DC;
        if (s > t) {
            sa[t][s] = 0.f;
            Pm[tid] = 0.f;
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
        for (int c = part * 4; c < dp; c += 16) {
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
                    for (int e = 0; e < 4; ++e) {      // (a pair above the diagonal is not kept; its power may not overflow)
                        const float w = yk[s][e] * power_of_2(fminf(xb[r][e] - yb[s][e], 0.f));
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
                    Pm[t * DC + u] = pq[r][s];
                }
            }
    }
    __syncthreads();
    // W and Y, a thread per column; what else the scan reads of a channel
    for (int j = tid; j < dp + p.dvp; j += 256) {
        float x[DC];
        if (j < dp) {
            const float last = sb[(DC - 1) * ld + j];
#pragma unroll
            for (int t = 0; t < DC; t += 4) {
                float kv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float b = sb[(t + i) * ld + j], k = sk[(t + i) * ld + j], e = power_of_2(b);
                    x[t + i] = k * e;
                    Qe[(size_t)(t + i) * dp + j] = sq[(t + i) * ld + j] * e;
                    kv[i] = k * power_of_2(last - b);
                }
                store4(Kt + (size_t)j * DC + t, kv);
            }
            E[j] = power_of_2(last);
        } else {
            const int c = j - dp;
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
        float* dst = j < dp ? W + j : Y + (j - dp);
        const int step = j < dp ? dp : p.dvp;
#pragma unroll
        for (int t = 0; t < DC; ++t) dst[(size_t)t * step] = x[t];
    }
}

__device__ __forceinline__ void dc_copy16(void* dst, const void* src, bool valid = true) {
    const int bytes = valid ? 16 : 0;      // 0: zeros, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
                 "r"(bytes) : "memory");
}

// A 32-bit number as two TF32 numbers.
struct Two { uint32_t hi, lo; };
__device__ __forceinline__ Two two_of(float x) {
    Two r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r.hi) : "f"(x));
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r.lo) : "f"(x - __uint_as_float(r.hi)));
    return r;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
                 "{%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// c += a b with both operands 32-bit; a: (row g, k 2t), (g + 8, 2t), (g, 2t + 1), (g + 8, 2t + 1); b: (k 2t, column g), (2t + 1, g)
__device__ __forceinline__ void mma_32(float (&c)[4], const Two (&a)[4], const Two (&b)[2]) {
    mma_tf32(c, a[0].lo, a[1].lo, a[2].lo, a[3].lo, b[0].hi, b[1].hi);
    mma_tf32(c, a[0].hi, a[1].hi, a[2].hi, a[3].hi, b[0].lo, b[1].lo);
    mma_tf32(c, a[0].hi, a[1].hi, a[2].hi, a[3].hi, b[0].hi, b[1].hi);
}
__device__ __forceinline__ void two_pair(Two (&b)[2], const float* p) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    b[0] = two_of(v.x);
    b[1] = two_of(v.y);
}

__host__ __device__ inline int dc_row(int dp) { return dp + (40 - dp % 32) % 32; }      // stride of a staged row of dp numbers

// Eight warps; a warp holds 16 NG channels of the state (dp <= 128 NG), transposed: S[j] is (column g or g + 8 of the block) x
// (channels 8 j + 2 t, 8 j + 2 t + 1), g = lane / 4, t = lane % 4.
template <int NG>
__global__ void __launch_bounds__(256) delta_chunk_scan_kernel(const DeltaChunkArgs p) {
    extern __shared__ __align__(16) float smem[];
    pdl_enter(TR_SCAN);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t2 = 2 * (lane & 3);
    const int h = blockIdx.y, col0 = blockIdx.x * DC;
    const int* por = p.portions + 4 * blockIdx.z;
    const int row0 = por[0], tokens = por[1], slot = por[2], chunk0 = por[3];
    if (slot < 0) return;
    const int dp = p.dp, ldw = dc_row(dp), chunks = (tokens + DC - 1) / DC;
    const int buf_floats = 2 * DC * ldw + dp * DC_KLD + dp + 2 * DC * DC;
    float* red = smem + 2 * buf_floats;     // [8 warps][16 columns][DC_RLD]: 32 sums over a warp's channels
    float* UT = red + 8 * DC * DC_RLD;      // [16 columns][DC_ULD]: U transposed
    float* OT = UT + DC * DC_ULD;           // the same of o's first part
    auto stage = [&](int i, int b) {
        const float* src = p.scratch + ((size_t)(chunk0 + i) * p.H + h) * p.stride;
        float* dst = smem + b * buf_floats;
        const int per = dp / 4;             // pieces of a row
        for (int x = tid; x < 2 * DC * per; x += 256) dc_copy16(dst + (x / per) * ldw + 4 * (x % per), src + 4 * (size_t)x);
        src += 2 * (size_t)DC * dp;
        dst += 2 * DC * ldw;
        for (int x = tid; x < dp * 4; x += 256) dc_copy16(dst + (x >> 2) * DC_KLD + 4 * (x & 3), src + 4 * (size_t)x);
        src += (size_t)dp * DC;
        dst += dp * DC_KLD;
        const int rest = (dp + DC * DC) / 4;
        for (int x = tid; x < rest; x += 256) dc_copy16(dst + 4 * x, src + 4 * (size_t)x);
        src += 4 * (size_t)rest;
        dst += 4 * rest;
        if (tid < DC * 4) {                 // this block's columns of Y
            const int t = tid >> 2, c = col0 + 4 * (tid & 3);
            const bool in = c < p.dvp;
            dc_copy16(dst + t * DC + 4 * (tid & 3), src + (size_t)t * p.dvp + (in ? c : 0), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    const int r0 = warp * 16 * NG;
    float* st = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
    float S[2 * NG][4];
#pragma unroll
    for (int j = 0; j < 2 * NG; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = r0 + 8 * j + t2 + (e & 1), c = col0 + g + 8 * (e >> 1);
            S[j][e] = r < p.d && c < p.dv ? st[(size_t)r * p.dv + c] : 0.f;
        }
    for (int i = 0; i < chunks; ++i) {
        const float* W = smem + (i & 1) * buf_floats;      // [32][ldw]: W, then q exp b
        const float* Kt = W + 2 * DC * ldw;
        const float* E = Kt + dp * DC_KLD;
        const float* Pm = E + dp;
        const float* Y = Pm + DC * DC;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                     // this chunk's numbers are there; the other buffer is free
        if (i + 1 < chunks) stage(i + 1, (i + 1) & 1);
        if (r0 < dp) {
            float acc[4][4];
#pragma unroll
            for (int x = 0; x < 4; ++x) acc[x][0] = acc[x][1] = acc[x][2] = acc[x][3] = 0.f;
#pragma unroll
            for (int j = 0; j < 2 * NG; ++j) {
                if (r0 + 8 * j >= dp) break;
                const Two a[4] = {two_of(S[j][0]), two_of(S[j][2]), two_of(S[j][1]), two_of(S[j][3])};
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    Two b[2];
                    two_pair(b, W + (8 * x + g) * ldw + r0 + 8 * j + t2);
                    mma_32(acc[x], a, b);
                }
            }
            float* mine = red + warp * DC * DC_RLD;
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                *reinterpret_cast<float2*>(mine + g * DC_RLD + 8 * x + t2) = make_float2(acc[x][0], acc[x][1]);
                *reinterpret_cast<float2*>(mine + (g + 8) * DC_RLD + 8 * x + t2) = make_float2(acc[x][2], acc[x][3]);
            }
        }
        __syncthreads();
        {   // the warps' sums in order: U = Y - W S (tokens 0 .. 15 of 32), o's first part (the others)
            const int c = tid >> 4, t = 2 * (tid & 15);
            float2 sum = make_float2(0.f, 0.f);
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                if (w * 16 * NG >= dp) break;
                const float2 v = *reinterpret_cast<const float2*>(red + w * DC * DC_RLD + c * DC_RLD + t);
                sum.x += v.x;
                sum.y += v.y;
            }
            if (t < DC)
                *reinterpret_cast<float2*>(UT + c * DC_ULD + t) = make_float2(Y[t * DC + c] - sum.x, Y[(t + 1) * DC + c] - sum.y);
            else
                *reinterpret_cast<float2*>(OT + c * DC_ULD + t - DC) = sum;
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
        for (int j = 0; j < 2 * NG; ++j) {
            if (r0 + 8 * j >= dp) break;
            const float2 e = *reinterpret_cast<const float2*>(E + r0 + 8 * j + t2);
            S[j][0] *= e.x; S[j][1] *= e.y; S[j][2] *= e.x; S[j][3] *= e.y;
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                Two b[2];
                two_pair(b, Kt + (r0 + 8 * j + g) * DC_KLD + 8 * x + t2);
                mma_32(S[j], u[x], b);
            }
        }
        if (warp >= 6) {                     // o: tokens 0 .. 7 and 8 .. 15
            const int t0 = 8 * (warp - 6);
            float2 lo = *reinterpret_cast<const float2*>(OT + g * DC_ULD + t0 + t2);
            float2 hi = *reinterpret_cast<const float2*>(OT + (g + 8) * DC_ULD + t0 + t2);
            float o[4] = {lo.x, lo.y, hi.x, hi.y};
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                Two b[2];
                two_pair(b, Pm + (t0 + g) * DC + 8 * x + t2);
                mma_32(o, u[x], b);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = i * DC + t0 + t2 + (e & 1), c = col0 + g + 8 * (e >> 1);
                if (t < tokens && c < p.dv) p.out[((size_t)(row0 + t) * p.H + h) * p.dv + c] = o[e];
            }
        }
    }
#pragma unroll
    for (int j = 0; j < 2 * NG; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = r0 + 8 * j + t2 + (e & 1), c = col0 + g + 8 * (e >> 1);
            if (r < p.d && c < p.dv) st[(size_t)r * p.dv + c] = S[j][e];
        }
}

}  // namespace air

// scratch: float32 [N, H, 3 * 16 dp + dp + 256 + 16 dvp] with dp = d filled up to a multiple of 16, dvp = dv to one of 4.
// Rows and slots as the lists say; d up to 256.
AIR_API int air_delta_portions(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* decay,
                               int ldd, const float* beta, int ldb, const float* a_log, const float* dt_bias, float* state,
                               float* out, const int* portions, int L, const int* chunks, int N, float* scratch, int H, int G,
                               int d, int dv, float q_scale, float unit_eps, cudaStream_t stream) {
    using namespace air;
    if (L <= 0 || N <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || d > DC_MAX_D || dv <= 0 || H > 65535 || L > 65535 || !scratch ||
        ((uintptr_t)scratch & 15))
        return AIR_ERR_BAD_ARGUMENT;
    DeltaChunkArgs a;
    a.q = q; a.ldq = ldq; a.k = k; a.ldk = ldk; a.v = v; a.ldv = ldv; a.decay = decay; a.ldd = ldd; a.beta = beta; a.ldb = ldb;
    a.a_log = a_log; a.dt_bias = dt_bias; a.chunks = chunks; a.portions = portions; a.scratch = scratch; a.state = state;
    a.out = out; a.H = H; a.G = G; a.d = d; a.dv = dv; a.dp = (d + 15) / 16 * 16; a.dvp = (dv + 3) / 4 * 4;
    a.q_scale = q_scale; a.unit_eps = unit_eps;
    a.stride = 3ll * a.dp * DC + a.dp + DC * DC + (long long)DC * a.dvp;
    const size_t smem1 = sizeof(float) * 3 * DC * (size_t)(a.dp + 4);
    if (smem1 > 44 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
        if (e != cudaSuccess) return (int)e;
    }
    int rc = launch(delta_chunk_prepare_kernel, dim3(N, H), 256, smem1, stream, a);
    if (rc) return rc;
    size_t smem2 = sizeof(float) * (2 * (size_t)(2 * DC * dc_row(a.dp) + a.dp * DC_KLD + a.dp + 2 * DC * DC) +
                                    8 * DC * DC_RLD + 2 * DC * DC_ULD);
    const dim3 grid((dv + DC - 1) / DC, H, L);
    // (as for the scan token by token: the blocks start when their predecessor has ended, and spread over the SMs)
    int sms = 148, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long blocks = (long long)grid.x * grid.y * grid.z;
    if (blocks <= sms && smem2 < 120 * 1024) smem2 = 120 * 1024;
    auto kernel = a.dp <= 128 ? delta_chunk_scan_kernel<1> : delta_chunk_scan_kernel<2>;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem2);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem2;
    cfg.stream = stream;
    return (int)cudaLaunchKernelEx(&cfg, kernel, a);
}

AIR_API int air_trace_set_delta_chunks(unsigned long long* buffer) { return air::set_trace_here(buffer); }
