// The matrix memory of mLSTM over the step's flat batch: every entry brings the next tokens of one request, rows
// q_start[e] .. q_start[e + 1], and slots[e] is the request's row of the states (negative: padding, skipped).  32-bit
// throughout.  x holds per token the projections q, k (H heads of d), v, g (H heads of dv), z one logit each for the input
// and the forget gate of every head, each at a column of its own.  Per head and token:
//
//   i = c tanh((zi + bi) / c),  f = log sigmoid(c tanh((zf + bf) / c)),  m' = max(f + m, i),
//   a = exp(f + m - m'),  b = exp(i - m'),
//   S = a S + b k v^T,  n = a n + b k,
//   o = S^T (q_scale q) / (max(|n . (q_scale q)|, exp(-m')) + 1e-6)
//   y = o / sqrt(mean(o^2) + eps) * w * sigmoid(g)      (the mean over the head's dv numbers, w [H * dv])
//
// with the states S [slots, H, d, dv], n [slots, H, d] and m [slots, H] zero at a request's start.
//
//   mlstm_step_kernel    one block per (head, entry) does all of it, token after token: the road of single next tokens (one
//                        launch behind the projections, the state read and written once) and of short portions.
//
// Longer portions are cut into chunks of ML_C tokens, counted from the portion's start.  With the decays a_t and weights
// b_t of the recurrence (they depend on the gates alone), P(s, t) = a_(s+1) .. a_t (products, not differences of sums of
// logarithms, so that a forgotten stretch costs no digits), W[t, s] = (q_t . k_s) b_s P(s, t) for s <= t inside a chunk and
// A_t = a_first .. a_t, a chunk's read-outs are W V + A (Q S_chunk) and n . q = row sum of W + A (q . n_chunk), with S_chunk
// and n_chunk the states ahead of the chunk: 32-bit products on the CUDA cores, rows of different chunks side by side.
//
//   mlstm_gates_kernel   a, b and exp(-m) of every token, its b P(t, end) and its A: block (head, portion); m by a parallel scan of the maps
//                        m -> max(F + m, M) (64-bit sums), 1,024 tokens at a time
//   mlstm_states_kernel  the states ahead of every chunk: block (tile of 32 x 64 of S, head, portion), the tile in
//                        registers, chunk after chunk: S <- (product of the chunk's a) S + sum_s b_s P(s, end) k_s v_s^T
//   mlstm_outputs_kernel block (chunk, head, 128 columns of v): the read-outs; where a head's v fits one block also the norm,
//                        the weight and the gate, else mlstm_finish_kernel does those
// A bfloat16 engine takes the same steps on the tensor cores (mlstm_tc.cu).
#include "mlstm.cuh"

namespace air {

__device__ __forceinline__ float ml_log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float ml_capped(float z, float cap) { return cap * tanhf(z / cap); }

// N: columns of S per access (4 where dv and the pointers allow it).
template <typename TX, typename TO, int N>
__global__ void __launch_bounds__(ML_THREADS) mlstm_step_kernel(const MlstmArgs p) {
    __shared__ float scratch[32];
    extern __shared__ __align__(16) float smem[];
    pdl_enter(TR_MLSTM);
    const int h = blockIdx.x, e = blockIdx.y, tid = threadIdx.x, d = p.d, dv = p.dv;
    const int slot = p.slots[e];
    if (slot < 0) return;
    const int q0 = p.q_start[e], cnt = p.q_start[e + 1] - q0;
    const int cols = dv / N, cw = min(cols, ML_THREADS), RG = ML_THREADS / cw;    // columns at a time, groups of rows
    const int rg = tid / cw, c_in = tid % cw;
    float *sk = smem, *sq = sk + d, *so = sq + d, *part = so + dv;                // part [RG][cw * N]
    float* S = p.S + ((size_t)slot * p.H + h) * d * dv;
    float* nn = p.n + ((size_t)slot * p.H + h) * d;
    float m = p.m[(size_t)slot * p.H + h];
    const float ib = p.ib[h], fb = p.fb[h];
    for (int t = 0; t < cnt; ++t) {
        const TX* row = (const TX*)p.x + (size_t)(q0 + t) * p.ldx;
        const float* zrow = p.z + (size_t)(q0 + t) * p.ldz;
        const float li = ml_capped(zrow[p.ci + h] + ib, p.cap);
        const float lf = ml_log_sigmoid(ml_capped(zrow[p.cf + h] + fb, p.cap));
        const float mn = fmaxf(lf + m, li);
        const float a = expf(lf + m - mn), b = expf(li - mn);
        m = mn;
        float nq = 0.f;
        for (int r = tid; r < d; r += ML_THREADS) {
            const float k = b * to_float(row[p.ck + h * d + r]), q = to_float(row[p.cq + h * d + r]) * p.q_scale;
            sk[r] = k;
            sq[r] = q;
            const float v = fmaf(a, nn[r], k);
            nn[r] = v;
            nq = fmaf(v, q, nq);
        }
        nq = block_sum(nq, scratch);                      // (its barriers also publish sk and sq)
        const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
        for (int c0 = 0; c0 < cols; c0 += cw) {
            const int c = c0 + c_in;
            float acc[N];
#pragma unroll
            for (int j = 0; j < N; ++j) acc[j] = 0.f;
            if (rg < RG && c < cols) {
                float v[N];
#pragma unroll
                for (int j = 0; j < N; ++j) v[j] = to_float(row[p.cv + h * dv + c * N + j]);
                float* col = S + (size_t)c * N;
                constexpr int U = 8;                      // rows of a thread under way at once
                for (int r0 = rg; r0 < d; r0 += U * RG) {
                    float s[U][N];
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        const int r = r0 + u * RG;
                        if (r < d) {
                            if constexpr (N == 4) load4(col + (size_t)r * dv, s[u]);
                            else s[u][0] = col[(size_t)r * dv];
                        }
                    }
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        const int r = r0 + u * RG;
                        if (r < d) {
                            const float k = sk[r], q = sq[r];
#pragma unroll
                            for (int j = 0; j < N; ++j) {
                                s[u][j] = fmaf(a, s[u][j], k * v[j]);
                                acc[j] = fmaf(s[u][j], q, acc[j]);
                            }
                            if constexpr (N == 4) store4(col + (size_t)r * dv, s[u]);
                            else col[(size_t)r * dv] = s[u][0];
                        }
                    }
                }
#pragma unroll
                for (int j = 0; j < N; ++j) part[(size_t)rg * cw * N + c_in * N + j] = acc[j];
            }
            __syncthreads();
            for (int x = tid; x < cw * N && c0 * N + x < dv; x += ML_THREADS) {
                float o = 0.f;
                for (int g = 0; g < RG; ++g) o += part[(size_t)g * cw * N + x];
                so[c0 * N + x] = o * inv;
            }
            __syncthreads();
        }
        float ss = 0.f;
        for (int c = tid; c < dv; c += ML_THREADS) ss = fmaf(so[c], so[c], ss);
        const float scale = 1.f / sqrtf(block_sum(ss, scratch) / (float)dv + p.eps);
        TO* y = (TO*)p.y + ((size_t)(q0 + t) * p.H + h) * dv;
        for (int c = tid; c < dv; c += ML_THREADS) {
            const float g = to_float(row[p.cg + h * dv + c]);
            y[c] = from_float<TO>(so[c] * scale * p.w[h * dv + c] / (1.f + expf(-g)));
        }
    }
    if (tid == 0) p.m[(size_t)slot * p.H + h] = m;
}

// ------------------------------------------------------------------ longer portions
constexpr int ML_TD = 32, ML_TV = 64;      // the tile of S that a block of mlstm_states_kernel holds
constexpr int ML_OV = 128;                 // columns of v per block of mlstm_outputs_kernel
constexpr int ML_KS = 64;                  // key channels staged at a time there
constexpr int ML_LD = ML_KS + 4, ML_LV = ML_OV + 4;

constexpr int ML_GT = 1024;                // threads of mlstm_gates_kernel

__global__ void __launch_bounds__(ML_GT) mlstm_gates_kernel(const MlstmChunkArgs c) {
    __shared__ double wF[ML_GT / 32], wM[ML_GT / 32], mt[ML_GT + 1];
    __shared__ float wP[ML_GT / 32];
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = c.p;
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int row0 = c.portions[blockIdx.y * 4], cnt = c.portions[blockIdx.y * 4 + 1], slot = c.portions[blockIdx.y * 4 + 2];
    const float ib = p.ib[h], fb = p.fb[h];
    double carry = (double)p.m[(size_t)slot * p.H + h];
    const size_t plane = (size_t)p.H * c.T;
    float* g = c.gates + (size_t)h * c.T + row0;
    auto logit = [&](int t, int col) { return t < cnt ? p.z[(size_t)(row0 + t) * p.ldz + col + h] : 0.f; };
    float zi = logit(tid, p.ci), zf = logit(tid, p.cf);
    for (int t0 = 0; t0 < cnt; t0 += ML_GT) {
        const int t = t0 + tid;
        // a place behind the portion's end leaves m as it is: F = 0, M far below
        float lf = 0.f, li = -1e30f;
        if (t < cnt) {
            li = ml_capped(zi + ib, p.cap);
            lf = ml_log_sigmoid(ml_capped(zf + fb, p.cap));
        }
        zi = logit(t + ML_GT, p.ci);       // (the next tokens' logits are on their way meanwhile)
        zf = logit(t + ML_GT, p.cf);
        double F = lf, M = li;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const double F0 = __shfl_up_sync(0xffffffffu, F, off), M0 = __shfl_up_sync(0xffffffffu, M, off);
            if (lane >= off) {
                M = fmax(M0 + F, M);
                F = F0 + F;
            }
        }
        if (lane == 31) { wF[warp] = F; wM[warp] = M; }
        if (tid == 0) mt[0] = carry;
        __syncthreads();
        if (warp == 0) {                   // the maps of all warps before each warp, by one more scan
            double F1 = wF[lane], M1 = wM[lane];
#pragma unroll
            for (int off = 1; off < 32; off <<= 1) {
                const double F0 = __shfl_up_sync(0xffffffffu, F1, off), M0 = __shfl_up_sync(0xffffffffu, M1, off);
                if (lane >= off) {
                    M1 = fmax(M0 + F1, M1);
                    F1 = F0 + F1;
                }
            }
            wF[lane] = F1;
            wM[lane] = M1;
        }
        __syncthreads();
        double m = warp == 0 ? carry : fmax(wF[warp - 1] + carry, wM[warp - 1]);
        m = fmax(F + m, M);
        mt[tid + 1] = m;
        __syncthreads();
        const float a = t < cnt ? expf((float)((double)lf + mt[tid] - m)) : 1.f;
        carry = mt[ML_GT];
        // products over the token's chunk (two warps): of everything up to it, and of everything behind it
        float upto = a, behind = a;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, upto, off), b = __shfl_down_sync(0xffffffffu, behind, off);
            if (lane >= off) upto *= u;
            if (lane + off < 32) behind *= b;
        }
        if (lane == 31) wP[warp] = upto;
        behind = __shfl_down_sync(0xffffffffu, behind, 1);
        if (lane == 31) behind = 1.f;
        __syncthreads();
        if (warp & 1) upto *= wP[warp - 1];
        else behind *= wP[warp + 1];
        if (t < cnt) {
            const float b = expf((float)((double)li - m));
            g[t] = a;
            g[plane + t] = b;
            g[2 * plane + t] = expf(-(float)m);
            g[3 * plane + t] = b * behind;
            g[4 * plane + t] = upto;
        }
        __syncthreads();
    }
    if (tid == 0) p.m[(size_t)slot * p.H + h] = (float)carry;
}

// The gates of L portions: what every road of portions starts with.
int launch_mlstm_gates(const MlstmChunkArgs& c, int L, cudaStream_t stream) {
    return launch(mlstm_gates_kernel, dim3(c.p.H, L), ML_GT, 0, stream, c);
}

__device__ __forceinline__ void ml_cp16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem)
                 : "memory");
}
__device__ __forceinline__ void ml_cp4(void* smem, const void* gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem)
                 : "memory");
}

// `rows` x COLS numbers from src (row stride ld, `width` columns of it exist, `live` rows exist) to dst (row stride DLD) by
// cp.async, zeros where there are none; NT threads.  vec: 16-byte pieces (everything a multiple of 4 numbers).
template <int COLS, int DLD, int NT>
__device__ __forceinline__ void ml_stage(float* dst, const float* src, size_t ld, int rows, int live, int width, int vec) {
    if (vec) {
        constexpr int P4 = COLS / 4;
        for (int i = threadIdx.x; i < rows * P4; i += NT) {
            const int r = i / P4, c = i % P4 * 4;
            float* to = dst + r * DLD + c;
            if (r < live && c < width) ml_cp16(to, src + (size_t)r * ld + c);
            else *reinterpret_cast<float4*>(to) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int i = threadIdx.x; i < rows * COLS; i += NT) {
            const int r = i / COLS, c = i % COLS;
            float* to = dst + r * DLD + c;
            if (r < live && c < width) ml_cp4(to, src + (size_t)r * ld + c);
            else *to = 0.f;
        }
    }
}

constexpr size_t ML_STATES_SMEM = sizeof(float) * 2 * (ML_C * (ML_TD + ML_TV) + ML_C + 4);

// 128 threads, 4 x 4 numbers of the tile each.
__global__ void __launch_bounds__(128) mlstm_states_kernel(const MlstmChunkArgs c) {
    extern __shared__ __align__(16) float smem[];
    constexpr int BUF = ML_C * (ML_TD + ML_TV) + ML_C + 4;       // a chunk: k, v, b P(s, end), the product of its a
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = c.p;
    const int d = p.d, dv = p.dv, tid = threadIdx.x, h = blockIdx.y;
    const int tiles_v = (dv + ML_TV - 1) / ML_TV;
    const int r0 = blockIdx.x / tiles_v * ML_TD, v0 = blockIdx.x % tiles_v * ML_TV;
    const int* po = c.portions + blockIdx.z * 4;
    const int row0 = po[0], cnt = po[1], slot = po[2], chunk0 = po[3];
    const int ty = tid >> 4, tx = tid & 15;
    const bool has_n = v0 == 0 && tid < ML_TD && r0 + tid < d;
    float acc[4][4], nacc = 0.f;
    float* S = p.S + ((size_t)slot * p.H + h) * d * dv;
    float* nn = p.n + ((size_t)slot * p.H + h) * d;
    const bool v4 = dv % 4 == 0 && v0 + tx * 4 < dv;       // (then the four columns exist and lie on 16 bytes)
    auto at = [&](float* base, int i) { return base + (size_t)(r0 + ty * 4 + i) * dv + v0 + tx * 4; };
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            acc[i][j] = (r0 + ty * 4 + i < d && v0 + tx * 4 + j < dv) ? at(S, i)[j] : 0.f;
    if (has_n) nacc = nn[r0 + tid];
    const size_t plane = (size_t)p.H * c.T;
    const float* ga = c.gates + (size_t)h * c.T + row0;
    auto stage = [&](int t0, int b) {
        const float* src = (const float*)p.x + (size_t)(row0 + t0) * p.ldx;
        float *sk = smem + b * BUF, *sv = sk + ML_C * ML_TD, *se = sv + ML_C * ML_TV;
        ml_stage<ML_TD, ML_TD, 128>(sk, src + p.ck + h * d + r0, p.ldx, ML_C, cnt - t0, d - r0, c.vec);
        ml_stage<ML_TV, ML_TV, 128>(sv, src + p.cv + h * dv + v0, p.ldx, ML_C, cnt - t0, dv - v0, c.vec);
        if (tid < ML_C) {
            if (t0 + tid < cnt) ml_cp4(se + tid, ga + 3 * plane + t0 + tid);
            else se[tid] = 0.f;
        } else if (tid == ML_C) {
            ml_cp4(se + ML_C, ga + 4 * plane + min(t0 + ML_C, cnt) - 1);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    int b = 0;
    for (int t0 = 0, ch = chunk0; t0 < cnt; t0 += ML_C, ++ch, b ^= 1) {
        // the states ahead of this chunk
        float* cs = c.chunk_S + ((size_t)ch * p.H + h) * d * dv;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            if (r0 + ty * 4 + i >= d) continue;
            if (v4) *reinterpret_cast<float4*>(at(cs, i)) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            else
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (v0 + tx * 4 + j < dv) at(cs, i)[j] = acc[i][j];
        }
        if (has_n) c.chunk_n[((size_t)ch * p.H + h) * d + r0 + tid] = nacc;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t0 + ML_C < cnt) stage(t0 + ML_C, b ^ 1);
        const float *sk = smem + b * BUF, *sv = sk + ML_C * ML_TD, *e = sv + ML_C * ML_TV;
        const float all = e[ML_C];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] *= all;
#pragma unroll 8
        for (int s = 0; s < ML_C; ++s) {
            float k[4], v[4];
            load4(sk + s * ML_TD + ty * 4, k);
            load4(sv + s * ML_TV + tx * 4, v);
            const float weight = e[s];
#pragma unroll
            for (int i = 0; i < 4; ++i) k[i] *= weight;
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(k[i], v[j], acc[i][j]);
        }
        if (has_n) {
            float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
            for (int s = 0; s < ML_C; s += 4)
#pragma unroll
                for (int j = 0; j < 4; ++j) part[j] = fmaf(e[s + j], sk[(s + j) * ML_TD + tid], part[j]);
            nacc = fmaf(nacc, all, (part[0] + part[1]) + (part[2] + part[3]));
        }
        // (the next round's barrier stands between these reads and the copies into this buffer after next)
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (r0 + ty * 4 + i < d && v0 + tx * 4 + j < dv) at(S, i)[j] = acc[i][j];
    if (has_n) nn[r0 + tid] = nacc;
}

// acc[i][j] += sum_k A[4 ty + i][k] B[k][4 tx + j (j < 4), 64 + 4 tx + j - 4]: A [64, ML_LD], B [64, ML_LV], 64 values of k
__device__ __forceinline__ void ml_product(float (&acc)[4][8], const float* A, const float* B, int ty, int tx) {
#pragma unroll 2
    for (int k0 = 0; k0 < 64; k0 += 4) {
        float a[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) load4(A + (4 * ty + i) * ML_LD + k0, a[i]);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            float b0[4], b1[4];
            load4(B + (k0 + kk) * ML_LV + 4 * tx, b0);
            load4(B + (k0 + kk) * ML_LV + 64 + 4 * tx, b1);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(a[i][kk], b0[j], acc[i][j]);
                    acc[i][4 + j] = fmaf(a[i][kk], b1[j], acc[i][4 + j]);
                }
        }
    }
}

constexpr size_t ML_OUT_SMEM = sizeof(float) * (3 * 64 * ML_LD + 64 * ML_LV + 3 * 64 + ML_KS);

template <typename TO>
__global__ void __launch_bounds__(256, 2) mlstm_outputs_kernel(const MlstmChunkArgs c) {
    extern __shared__ __align__(16) float smem[];
    float *sq = smem, *sk = sq + 64 * ML_LD, *sw = sk + 64 * ML_LD, *sb = sw + 64 * ML_LD;
    float *sa = sb + 64 * ML_LV, *sA = sa + 64, *sinv = sA + 64, *sn = sinv + 64;
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = c.p;
    const int ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * ML_OV, tid = threadIdx.x, d = p.d, dv = p.dv;
    const int row0 = c.chunks[2 * ch], cnt = c.chunks[2 * ch + 1];
    const int ty = tid >> 4, tx = tid & 15;
    const float *ga = c.gates + (size_t)h * c.T + row0, *gb = ga + (size_t)p.H * c.T, *ge = gb + (size_t)p.H * c.T;
    const float* src = (const float*)p.x + (size_t)row0 * p.ldx;
    const float* S = c.chunk_S + ((size_t)ch * p.H + h) * d * dv;
    const float* nn = c.chunk_n + ((size_t)ch * p.H + h) * d;
    auto stage = [&](int k0) {
        ml_stage<ML_KS, ML_LD, 256>(sq, src + p.cq + h * d + k0, p.ldx, 64, cnt, d - k0, c.vec);
        ml_stage<ML_KS, ML_LD, 256>(sk, src + p.ck + h * d + k0, p.ldx, 64, cnt, d - k0, c.vec);
        ml_stage<ML_OV, ML_LV, 256>(sb, S + (size_t)k0 * dv + v0, dv, 64, d - k0, dv - v0, dv % 4 == 0);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (tid < ML_KS) sn[tid] = k0 + tid < d ? nn[k0 + tid] : 0.f;
    };
    stage(0);
    if (tid < 64) sa[tid] = tid < cnt ? ga[tid] : 1.f;
    __syncthreads();
    if (tid < 64) {          // b_s P(s, t) in the place of W[t, s]
        float w = tid < cnt ? gb[tid] : 0.f;
        for (int t = 0; t < 64; ++t) {
            if (t > tid) w *= sa[t];
            sw[t * ML_LD + tid] = t < tid ? 0.f : w;
        }
    } else if (tid < 128) {
        sA[tid - 64] = tid - 64 < cnt ? ga[4 * (size_t)p.H * c.T + tid - 64] : 0.f;
    }
    float acc[4][8], w[4][4], qn = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) w[i][j] = 0.f;
    }
    for (int k0 = 0; k0 < d; k0 += ML_KS) {
        if (k0) {
            __syncthreads();                               // the last slab has been used
            stage(k0);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // w[i][j] += q_(4 ty + i) . k_(tx + 16 j)
#pragma unroll 4
        for (int k = 0; k < ML_KS; k += 4) {
            float a[4][4], b[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) load4(sq + (4 * ty + i) * ML_LD + k, a[i]);
#pragma unroll
            for (int j = 0; j < 4; ++j) load4(sk + (tx + 16 * j) * ML_LD + k, b[j]);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk) w[i][j] = fmaf(a[i][kk], b[j][kk], w[i][j]);
        }
        ml_product(acc, sq, sb, ty, tx);
        // a quarter of q_t . n for row t = tid / 4
        const float* qr = sq + (tid >> 2) * ML_LD + (tid & 3) * 16;
        const float* nr = sn + (tid & 3) * 16;
#pragma unroll
        for (int k = 0; k < 16; ++k) qn = fmaf(qr[k], nr[k], qn);
    }
    __syncthreads();
    // the values take the last slab's place
    ml_stage<ML_OV, ML_LV, 256>(sb, src + p.cv + h * dv + v0, p.ldx, 64, cnt, dv - v0, c.vec);
    asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float A = sA[4 * ty + i];
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] *= A;
#pragma unroll
        for (int j = 0; j < 4; ++j) sw[(4 * ty + i) * ML_LD + tx + 16 * j] *= w[i][j];
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    {
        const int t = tid >> 2;
        const float* wr = sw + t * ML_LD + (tid & 3) * 16;
        float sum = sA[t] * qn;
#pragma unroll
        for (int k = 0; k < 16; ++k) sum += wr[k];
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if ((tid & 3) == 0)       // (q's scale multiplies both read-outs, here)
            sinv[t] = p.q_scale / (fmaxf(fabsf(sum * p.q_scale), t < cnt ? ge[t] : 1.f) + 1e-6f);
    }
    ml_product(acc, sw, sb, ty, tx);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        const float inv = sinv[t];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            acc[i][j] *= inv;
            ss = fmaf(acc[i][j], acc[i][j], ss);
        }
        auto column = [&](int j) { return v0 + (j < 4 ? 4 * tx + j : 64 + 4 * tx + j - 4); };
        if (c.o) {
            if (t < cnt)
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (column(j) < dv) c.o[((size_t)(row0 + t) * p.H + h) * dv + column(j)] = acc[i][j];
            continue;
        }
        // (columns beyond dv are zeros: they add nothing to the sum)
#pragma unroll
        for (int off = 1; off < 16; off <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        if (t >= cnt) continue;
        const float scale = 1.f / sqrtf(ss / (float)dv + p.eps);
        const float* gr = src + (size_t)t * p.ldx + p.cg + h * dv;
        TO* y = (TO*)p.y + ((size_t)(row0 + t) * p.H + h) * dv;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int col = column(j);
            if (col < dv) y[col] = from_float<TO>(acc[i][j] * scale * p.w[h * dv + col] / (1.f + expf(-gr[col])));
        }
    }
}

}  // namespace air

AIR_API int air_mlstm_step(const void* x, int x_dtype, int ldx, int cq, int ck, int cv, int cg, const float* z, int ldz, int ci,
                           int cf, const float* ib, const float* fb, const float* w, float* S, float* n, float* m, void* y,
                           int out_dtype, const int* q_start, const int* slots, int entries, int H, int d, int dv, float cap,
                           float q_scale, float eps, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (H <= 0 || d <= 0 || dv <= 0 || entries > 65535 || !(cap > 0.f)) return AIR_ERR_BAD_ARGUMENT;
    air::MlstmArgs p{x, ldx, z, ldz, cq, ck, cv, cg, ci, cf, ib, fb, w, S, n, m, y, q_start, slots, H, d, dv, cap, q_scale, eps};
    const bool vec = dv % 4 == 0 && ((uintptr_t)S & 15) == 0;
    const int N = vec ? 4 : 1, cols = dv / N, cw = cols < air::ML_THREADS ? cols : air::ML_THREADS;
    const size_t smem = sizeof(float) * ((size_t)2 * d + dv + (size_t)(air::ML_THREADS / cw) * cw * N);
    if (smem > 200 * 1024) return AIR_ERR_BAD_ARGUMENT;
    AIR_DISPATCH(x_dtype, TX, AIR_DISPATCH(out_dtype, TO, {
        auto go = [&](auto kernel) {
            if (smem > 44 * 1024) {
                cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                if (err != cudaSuccess) return (int)err;
            }
            return air::launch(kernel, dim3(H, entries), air::ML_THREADS, smem, stream, p);
        };
        return vec ? go(air::mlstm_step_kernel<TX, TO, 4>) : go(air::mlstm_step_kernel<TX, TO, 1>);
    }));
    return 0;
}

// Portions of several tokens (see the file's head): portions int32 [L, 4] = (first row, tokens, slot, first chunk) and
// chunks int32 [N, 2] = (first row, tokens), a portion's chunks of 64 tokens one after the other.  Scratch: gates float32
// [5, H, T], chunk_S [N, H, d, dv], chunk_n [N, H, d], and o [T, H, dv] where dv > 128.
AIR_API int air_mlstm_portions(const float* x, int ldx, int cq, int ck, int cv, int cg, const float* z, int ldz, int ci, int cf,
                               const float* ib, const float* fb, const float* w, float* S, float* n, float* m, void* y,
                               int out_dtype, const int* portions, int L, const int* chunks, int N, float* gates,
                               float* chunk_S, float* chunk_n, float* o, int T, int H, int d, int dv, float cap,
                               float q_scale, float eps, cudaStream_t stream) {
    if (L <= 0 || N <= 0) return 0;
    const int v_blocks = (dv + air::ML_OV - 1) / air::ML_OV;
    if (H <= 0 || H > 65535 || d <= 0 || dv <= 0 || L > 65535 || v_blocks > 65535 || !(cap > 0.f) || !gates || !chunk_S ||
        !chunk_n || (v_blocks > 1 && !o) || (((uintptr_t)chunk_S | (uintptr_t)S) & 15))
        return AIR_ERR_BAD_ARGUMENT;
    const int vec = ((ldx | cq | ck | cv | d | dv) & 3) == 0 && ((uintptr_t)x & 15) == 0;
    air::MlstmChunkArgs c;
    c.p = air::MlstmArgs{x, ldx, z, ldz, cq, ck, cv, cg, ci, cf, ib, fb, w, S, n, m, y, nullptr, nullptr, H, d, dv, cap, q_scale, eps};
    c.portions = portions; c.chunks = chunks; c.gates = gates; c.chunk_S = chunk_S; c.chunk_n = chunk_n;
    c.o = v_blocks > 1 ? o : nullptr; c.T = T; c.vec = vec;
    int rc = air::launch_mlstm_gates(c, L, stream);
    if (rc) return rc;
    const int tiles = ((d + air::ML_TD - 1) / air::ML_TD) * ((dv + air::ML_TV - 1) / air::ML_TV);
    // A block's time is a chain over its chunks, and blocks that share an SM stretch one another's.  Launched while the
    // kernel before it is still leaving the SMs they would land several to an SM, so this kernel starts when its
    // predecessor has ended, and while there are no more blocks than SMs (than twice the SMs) a block asks for so much
    // shared memory that only one (two) of them fit an SM.
    int sms = 148, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long blocks = (long long)tiles * H * L;
    const size_t smem = blocks <= sms ? 120 * 1024 : blocks <= 2ll * sms ? 80 * 1024 : air::ML_STATES_SMEM;
    cudaError_t err = cudaFuncSetAttribute(air::mlstm_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles, H, L);
    cfg.blockDim = dim3(128);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    rc = (int)cudaLaunchKernelEx(&cfg, air::mlstm_states_kernel, c);
    if (rc) return rc;
    AIR_DISPATCH(out_dtype, TO, {
        auto kernel = air::mlstm_outputs_kernel<TO>;
        err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)air::ML_OUT_SMEM);
        if (err != cudaSuccess) return (int)err;
        rc = air::launch(kernel, dim3(N, H, v_blocks), 256, air::ML_OUT_SMEM, stream, c);
        if (rc || v_blocks == 1) return rc;
        return air::launch(air::mlstm_finish_kernel<float, TO>, dim3(N, H), 128, 0, stream, c);
    });
    return 0;
}

AIR_API int air_trace_set_mlstm(unsigned long long* buffer) { return air::set_trace_here(buffer); }
