// The matrix memory of mLSTM over the step's flat batch: every entry brings the next tokens of one request, rows
// q_start[e] .. q_start[e + 1], and slots[e] is the request's row of the states (negative: padding, skipped).  32-bit
// throughout.  proj [T, ld] holds per token the projections q, k (H heads of d), v, g (H heads of dv) and one logit each
// for the input and the forget gate of every head, each at a column of its own.  Per head and token:
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
#include "common.cuh"

namespace air {

constexpr int ML_THREADS = 256;

struct MlstmArgs {
    const float* proj; int ld;
    int cq, ck, cv, cg, ci, cf;        // the columns at which the projections start
    const float* ib; const float* fb;  // [H]
    const float* w;                    // [H * dv]
    float* S; float* n; float* m;
    void* y;                           // [T, H * dv]
    const int* q_start; const int* slots;
    int H, d, dv;
    float cap, q_scale, eps;
};

__device__ __forceinline__ float ml_log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float ml_capped(float z, float cap) { return cap * tanhf(z / cap); }

// N: columns of S per access (4 where dv and the pointers allow it).
template <typename TO, int N>
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
        const float* row = p.proj + (size_t)(q0 + t) * p.ld;
        const float li = ml_capped(row[p.ci + h] + ib, p.cap);
        const float lf = ml_log_sigmoid(ml_capped(row[p.cf + h] + fb, p.cap));
        const float mn = fmaxf(lf + m, li);
        const float a = expf(lf + m - mn), b = expf(li - mn);
        m = mn;
        float nq = 0.f;
        for (int r = tid; r < d; r += ML_THREADS) {
            const float k = b * row[p.ck + h * d + r], q = row[p.cq + h * d + r] * p.q_scale;
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
                for (int j = 0; j < N; ++j) v[j] = row[p.cv + h * dv + c * N + j];
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
            const float g = row[p.cg + h * dv + c];
            y[c] = from_float<TO>(so[c] * scale * p.w[h * dv + c] / (1.f + expf(-g)));
        }
    }
    if (tid == 0) p.m[(size_t)slot * p.H + h] = m;
}

}  // namespace air

AIR_API int air_mlstm_step(const float* proj, int ld, int cq, int ck, int cv, int cg, int ci, int cf, const float* ib,
                           const float* fb, const float* w, float* S, float* n, float* m, void* y, int out_dtype,
                           const int* q_start, const int* slots, int entries, int H, int d, int dv, float cap, float q_scale,
                           float eps, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (H <= 0 || d <= 0 || dv <= 0 || entries > 65535 || !(cap > 0.f)) return AIR_ERR_BAD_ARGUMENT;
    air::MlstmArgs p{proj, ld, cq, ck, cv, cg, ci, cf, ib, fb, w, S, n, m, y, q_start, slots, H, d, dv, cap, q_scale, eps};
    const bool vec = dv % 4 == 0 && ((uintptr_t)S & 15) == 0;
    const int N = vec ? 4 : 1, cols = dv / N, cw = cols < air::ML_THREADS ? cols : air::ML_THREADS;
    const size_t smem = sizeof(float) * ((size_t)2 * d + dv + (size_t)(air::ML_THREADS / cw) * cw * N);
    if (smem > 200 * 1024) return AIR_ERR_BAD_ARGUMENT;
    AIR_DISPATCH(out_dtype, TO, {
        auto go = [&](auto kernel) {
            if (smem > 44 * 1024) {
                cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                if (err != cudaSuccess) return (int)err;
            }
            return air::launch(kernel, dim3(H, entries), air::ML_THREADS, smem, stream, p);
        };
        return vec ? go(air::mlstm_step_kernel<TO, 4>) : go(air::mlstm_step_kernel<TO, 1>);
    });
    return 0;
}

AIR_API int air_trace_set_mlstm(unsigned long long* buffer) { return air::set_trace_here(buffer); }
