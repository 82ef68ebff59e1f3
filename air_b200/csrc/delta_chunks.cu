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
// delta_chunk_prepare_kernel   all that does not depend on the state, a block per chunk and head
// delta_chunk_scan_kernel      the last three lines, a block per head, portion and 16 columns of the state, which stays in
//                              shared memory; the next chunk's numbers arrive (cp.async) while this one's are used
//
// Everything is 32-bit (multiply-adds on the CUDA cores).  What a row is depends on the state and the portion's tokens only.
#include "common.cuh"

namespace air {

constexpr int DC = 16;              // tokens of a chunk, and columns of a block of the scan
constexpr int DC_LD = DC + 4;       // a staged row of 16 numbers: eight rows fall into different banks
constexpr int DC_MAX_D = 256;
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
    int H, G, d, dv, dp, dvp;       // dp: d filled up to a multiple of 8, dvp: dv to one of 4
    float q_scale, unit_eps;
    long long stride;               // of a chunk and head: W^T, (q exp b)^T [dp, 16] each, k exp(b_last - b) [16, dp],
                                    // exp b_last [dp], p [16, 16], Y [16, dvp]
};

__device__ __forceinline__ float softplus_1(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__global__ void __launch_bounds__(256) delta_chunk_prepare_kernel(const DeltaChunkArgs p) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float sa[DC][DC], sbeta[DC], kf[DC], qf[DC];
    pdl_enter(TR_SCAN);
    const int h = blockIdx.y, g = h / (p.H / p.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int q0 = p.chunks[2 * blockIdx.x], n = p.chunks[2 * blockIdx.x + 1];
    const int d = p.d, dp = p.dp, ld = dp + 4;
    float* sk = smem;                       // [16][ld]
    float* sq = sk + DC * ld;
    float* sb = sq + DC * ld;               // the decays' logarithms to the base 2, then their sums
    const float rate = -expf(p.a_log[h]) * 1.4426950408889634f;
    for (int idx = tid; idx < DC * dp; idx += 256) {
        const int t = idx / dp, c = idx % dp;
        float k = 0.f, q = 0.f, b = 0.f;
        if (t < n && c < d) {
            k = p.k[(size_t)(q0 + t) * p.ldk + g * d + c];
            q = p.q[(size_t)(q0 + t) * p.ldq + g * d + c];
            b = fmaxf(rate * softplus_1(p.decay[(size_t)(q0 + t) * p.ldd + h * d + c] + p.dt_bias[h * d + c]), DC_FLOOR);
        }
        sk[t * ld + c] = k;
        sq[t * ld + c] = q;
        sb[t * ld + c] = b;
    }
    if (tid < DC) sbeta[tid] = tid < n ? 1.f / (1.f + expf(-p.beta[(size_t)(q0 + tid) * p.ldb + h])) : 0.f;
    __syncthreads();
    for (int t = warp; t < DC; t += 8) {    // lengths
        float ss = 0.f, qs = 0.f;
        for (int c = lane; c < d; c += 32) {
            ss = fmaf(sk[t * ld + c], sk[t * ld + c], ss);
            qs = fmaf(sq[t * ld + c], sq[t * ld + c], qs);
        }
        ss = warp_sum(ss);
        qs = warp_sum(qs);
        if (lane == 0) {
            kf[t] = 1.f / sqrtf(ss + p.unit_eps);
            qf[t] = p.q_scale / sqrtf(qs + p.unit_eps);
        }
    }
    for (int c = tid; c < dp; c += 256) {
        float sum = 0.f;
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            sum += sb[t * ld + c];
            sb[t * ld + c] = sum;
        }
    }
    __syncthreads();
    for (int idx = tid; idx < DC * dp; idx += 256) {
        const int t = idx / dp, c = idx % dp;
        sk[t * ld + c] *= kf[t];
        sq[t * ld + c] *= qf[t];
    }
    __syncthreads();
    float* base = p.scratch + ((size_t)blockIdx.x * p.H + h) * p.stride;
    float* Wt = base;
    float* Qt = Wt + (size_t)dp * DC;
    float* Kh = Qt + (size_t)dp * DC;
    float* E = Kh + (size_t)DC * dp;
    float* Pm = E + dp;
    float* Y = Pm + DC * DC;
    {   // a and p: a thread per pair of tokens
        const int t = tid / DC, s = tid % DC;
        float a = 0.f, pq = 0.f;
        if (s <= t) {
            const float *kt = sk + t * ld, *qt = sq + t * ld, *ks = sk + s * ld, *bt = sb + t * ld, *bs = sb + s * ld;
            for (int c = 0; c < dp; c += 4) {
                float xk[4], xq[4], xs[4], xb[4], yb[4];
                load4(kt + c, xk);
                load4(qt + c, xq);
                load4(ks + c, xs);
                load4(bt + c, xb);
                load4(bs + c, yb);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float e = xs[j] * exp2f(xb[j] - yb[j]);
                    a = fmaf(xk[j], e, a);
                    pq = fmaf(xq[j], e, pq);
                }
            }
        }
        sa[t][s] = s < t ? sbeta[t] * a : 0.f;
        Pm[tid] = pq;
    }
    __syncthreads();
    // W and Y, a thread per column; what else the scan reads of a channel
    for (int j = tid; j < dp + p.dvp; j += 256) {
        float x[DC];
        if (j < dp) {
            float e[DC];
#pragma unroll
            for (int t = 0; t < DC; ++t) {
                e[t] = exp2f(sb[t * ld + j]);
                x[t] = sk[t * ld + j] * e[t];
            }
            const float last = sb[(DC - 1) * ld + j];
#pragma unroll
            for (int t = 0; t < DC; t += 4) {
                float qv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    qv[i] = sq[(t + i) * ld + j] * e[t + i];
                    Kh[(size_t)(t + i) * dp + j] = sk[(t + i) * ld + j] * exp2f(last - sb[(t + i) * ld + j]);
                }
                store4(Qt + (size_t)j * DC + t, qv);
            }
            E[j] = e[DC - 1];
        } else {
            const int c = j - dp;
#pragma unroll
            for (int t = 0; t < DC; ++t) x[t] = t < n && c < p.dv ? p.v[(size_t)(q0 + t) * p.ldv + h * p.dv + c] : 0.f;
        }
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            float sum = sbeta[t] * x[t];
#pragma unroll
            for (int s = 0; s < t; ++s) sum = fmaf(-sa[t][s], x[s], sum);
            x[t] = sum;
        }
        if (j < dp) {
#pragma unroll
            for (int t = 0; t < DC; t += 4) {
                const float w[4] = {x[t], x[t + 1], x[t + 2], x[t + 3]};
                store4(Wt + (size_t)j * DC + t, w);
            }
        } else {
#pragma unroll
            for (int t = 0; t < DC; ++t) Y[(size_t)t * p.dvp + (j - dp)] = x[t];
        }
    }
}

__device__ __forceinline__ void dc_copy16(void* dst, const void* src, bool valid = true) {
    const int bytes = valid ? 16 : 0;      // 0: zeros, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
                 "r"(bytes) : "memory");
}

__global__ void __launch_bounds__(256) delta_chunk_scan_kernel(const DeltaChunkArgs p) {
    extern __shared__ __align__(16) float smem[];
    pdl_enter(TR_SCAN);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, col0 = blockIdx.x * DC;
    const int* por = p.portions + 4 * blockIdx.z;
    const int row0 = por[0], tokens = por[1], slot = por[2], chunk0 = por[3];
    if (slot < 0) return;
    const int dp = p.dp, chunks = (tokens + DC - 1) / DC;
    const int buf_floats = 2 * dp * DC_LD + DC * dp + dp + 2 * DC * DC;
    float* S = smem + 2 * buf_floats;       // [dp][16]
    float* U = S + dp * DC;                 // [16][16]
    auto stage = [&](int i, int b) {
        const float* src = p.scratch + ((size_t)(chunk0 + i) * p.H + h) * p.stride;
        float* dst = smem + b * buf_floats;
        for (int x = tid; x < 2 * dp * 4; x += 256)           // W^T and (q exp b)^T, rows of 16
            dc_copy16(dst + (x >> 2) * DC_LD + 4 * (x & 3), src + 4 * (size_t)x);
        src += 2 * (size_t)dp * DC;
        dst += 2 * dp * DC_LD;
        const int rest = (DC * dp + dp + DC * DC) / 4;        // k exp(b_last - b), exp b_last, p as they lie
        for (int x = tid; x < rest; x += 256) dc_copy16(dst + 4 * x, src + 4 * (size_t)x);
        src += 4 * (size_t)rest;
        dst += 4 * rest;
        if (tid < DC * 4) {                                   // this block's columns of Y
            const int t = tid >> 2, c = col0 + 4 * (tid & 3);
            const bool in = c < p.dvp;
            dc_copy16(dst + t * DC + 4 * (tid & 3), src + (size_t)t * p.dvp + (in ? c : 0), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    float* st = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
    for (int idx = tid; idx < dp * DC; idx += 256) {
        const int r = idx / DC, c = col0 + idx % DC;
        S[idx] = r < p.d && c < p.dv ? st[(size_t)r * p.dv + c] : 0.f;
    }
    // U and o's first part: warps 0-3 take W, warps 4-7 q exp b, four rows each; a lane takes four columns and an eighth of
    // the channels
    const int which = warp >> 2, tt = warp & 3, ct = lane & 3, kq = lane >> 2;
    const int b4 = lane >> 4 & 1, b3 = lane >> 3 & 1, b2 = lane >> 2 & 1;
    const int row = tt * 4 + 2 * b4 + b3, col = ct * 4 + 2 * b2;      // the two sums that stay with this lane
    for (int i = 0; i < chunks; ++i) {
        const float* buf = smem + (i & 1) * buf_floats;
        const float* M = buf + which * dp * DC_LD;
        const float* Kh = buf + 2 * dp * DC_LD;
        const float* E = Kh + DC * dp;
        const float* Pm = E + dp;
        const float* Y = Pm + DC * DC;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                     // this chunk's numbers and the state are there; the other buffer is free
        if (i + 1 < chunks) stage(i + 1, (i + 1) & 1);
        float acc[4][4];
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[a][c] = 0.f;
#pragma unroll 4
        for (int k = kq; k < dp; k += 8) {
            float m[4], s[4];
            load4(M + k * DC_LD + tt * 4, m);
            load4(S + k * DC + ct * 4, s);
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int c = 0; c < 4; ++c) acc[a][c] = fmaf(m[a], s[c], acc[a][c]);
        }
        // the eight lanes' sums: each exchange halves what a lane holds
        float r2[2][4], r1[4], r0[2];
#pragma unroll
        for (int a = 0; a < 2; ++a)
#pragma unroll
            for (int c = 0; c < 4; ++c)
                r2[a][c] = (b4 ? acc[a + 2][c] : acc[a][c]) + __shfl_xor_sync(0xffffffffu, b4 ? acc[a][c] : acc[a + 2][c], 16);
#pragma unroll
        for (int c = 0; c < 4; ++c)
            r1[c] = (b3 ? r2[1][c] : r2[0][c]) + __shfl_xor_sync(0xffffffffu, b3 ? r2[0][c] : r2[1][c], 8);
#pragma unroll
        for (int c = 0; c < 2; ++c)
            r0[c] = (b2 ? r1[c + 2] : r1[c]) + __shfl_xor_sync(0xffffffffu, b2 ? r1[c] : r1[c + 2], 4);
        if (which == 0) {
            U[row * DC + col] = Y[row * DC + col] - r0[0];
            U[row * DC + col + 1] = Y[row * DC + col + 1] - r0[1];
        }
        __syncthreads();
        if (which == 1) {
#pragma unroll
            for (int s = 0; s < DC; ++s) {
                const float w = Pm[row * DC + s];
                const float2 u = *reinterpret_cast<const float2*>(U + s * DC + col);
                r0[0] = fmaf(w, u.x, r0[0]);
                r0[1] = fmaf(w, u.y, r0[1]);
            }
            const int t = i * DC + row;
            if (t < tokens) {
                float* o = p.out + ((size_t)(row0 + t) * p.H + h) * p.dv + col0 + col;
                if (col0 + col < p.dv) o[0] = r0[0];
                if (col0 + col + 1 < p.dv) o[1] = r0[1];
            }
        }
        // the state: a thread takes four columns of every 64th channel
        for (int k = tid >> 2; k < dp; k += 64) {
            const int c = (tid & 3) * 4;
            float s[4];
            load4(S + k * DC + c, s);
            const float e = E[k];
#pragma unroll
            for (int j = 0; j < 4; ++j) s[j] *= e;
#pragma unroll
            for (int t = 0; t < DC; ++t) {
                float u[4];
                load4(U + t * DC + c, u);
                const float kk = Kh[t * dp + k];
#pragma unroll
                for (int j = 0; j < 4; ++j) s[j] = fmaf(kk, u[j], s[j]);
            }
            store4(S + k * DC + c, s);
        }
    }
    __syncthreads();
    for (int idx = tid; idx < dp * DC; idx += 256) {
        const int r = idx / DC, c = col0 + idx % DC;
        if (r < p.d && c < p.dv) st[(size_t)r * p.dv + c] = S[idx];
    }
}

}  // namespace air

// Floats of scratch per chunk and head.
AIR_API long long air_delta_chunk_stride(int d, int dv) {
    const long long dp = (d + 7) / 8 * 8, dvp = (dv + 3) / 4 * 4;
    return 3 * dp * air::DC + dp + air::DC * air::DC + air::DC * dvp;
}

// scratch: float32 [N, H, air_delta_chunk_stride(d, dv)].  Rows and slots as the lists say; d up to 256.
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
    a.out = out; a.H = H; a.G = G; a.d = d; a.dv = dv; a.dp = (d + 7) / 8 * 8; a.dvp = (dv + 3) / 4 * 4;
    a.q_scale = q_scale; a.unit_eps = unit_eps; a.stride = air_delta_chunk_stride(d, dv);
    const size_t smem1 = sizeof(float) * 3 * DC * (size_t)(a.dp + 4);
    if (smem1 > 44 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
        if (e != cudaSuccess) return (int)e;
    }
    int rc = launch(delta_chunk_prepare_kernel, dim3(N, H), 256, smem1, stream, a);
    if (rc) return rc;
    size_t smem2 = sizeof(float) * (2 * (size_t)(2 * a.dp * DC_LD + DC * a.dp + a.dp + 2 * DC * DC) + a.dp * DC + DC * DC);
    const dim3 grid((dv + DC - 1) / DC, H, L);
    // (as for the scan token by token: the blocks start when their predecessor has ended, and spread over the SMs)
    int sms = 148, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long blocks = (long long)grid.x * grid.y * grid.z;
    if (blocks <= sms && smem2 < 120 * 1024) smem2 = 120 * 1024;
    else if (blocks <= 2ll * sms && smem2 < 80 * 1024) smem2 = 80 * 1024;
    cudaError_t e = cudaFuncSetAttribute(delta_chunk_scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem2);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem2;
    cfg.stream = stream;
    return (int)cudaLaunchKernelEx(&cfg, delta_chunk_scan_kernel, a);
}

AIR_API int air_trace_set_delta_chunks(unsigned long long* buffer) { return air::set_trace_here(buffer); }
