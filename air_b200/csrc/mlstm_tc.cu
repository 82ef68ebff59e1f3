// Longer portions of mLSTM's matrix memory in a bfloat16 engine: the chunks of mlstm.cu with their products on the tensor
// cores (mma.sync m16n8k16, 32-bit sums).  q, k, v and the output gate's logits come in bfloat16, straight from their
// product; everything that enters the recurrence is 32-bit: gates, decays, m, n and S are, and where a 32-bit number is
// an operand of a product (a weighted key, a chunk's weights W, a state S) it enters as the sum of two bfloat16 numbers.
//
//   mlstm_gates_kernel        as for the other road (mlstm.cu)
//   mlstm_tc_update_kernel    U = sum_s (b_s P(s, end) k_s) v_s^T and the like sum of k alone, for every chunk, side by side:
//                             block (tile of 64 x 128, head, chunk)
//   mlstm_tc_chain_kernel     the states ahead of every chunk, S <- (product of the chunk's a) S + U: a thread takes four
//                             numbers of S through all chunks of a portion, and writes them as two bfloat16 planes
//   mlstm_tc_outputs_kernel   block (chunk, head, 128 columns of v), a warp per 16 tokens: W = (Q K^T) times the decays (in
//                             registers), A (Q S) + W V, the denominator, and where a head's v fits one block the norm, the
//                             weight and the gate; else mlstm_finish_kernel does those
#include "mlstm.cuh"
#include "mma.cuh"

namespace air {

struct MlstmTcArgs {
    MlstmChunkArgs c;                  // c.p.x in bfloat16
    float* U;                          // [N, H, d, dv]
    __nv_bfloat16* S2;                 // [N, H, 2, d, dv]: the states ahead of every chunk, high part and rest
};

constexpr int MT_LK = 72, MT_LV = 136;     // row lengths in shared memory (64 and 128 numbers; 8 rows on different banks)
constexpr int MT_LD = 68;
static_assert(64 * MT_LV <= 2 * 64 * MT_LK, "the gate's rows fit where q and k were");

__device__ __forceinline__ uint32_t mt_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// 64 rows of COLS bfloat16 numbers from src (row stride ld; `live` rows and `width` columns exist, the others are zeros) to
// rows of LD numbers, by 128 threads with cp.async
template <int COLS, int LD>
__device__ __forceinline__ void mt_stage(__nv_bfloat16* dst, const __nv_bfloat16* src, size_t ld, int live, int width) {
    constexpr int P8 = COLS / 8;
    for (int i = threadIdx.x; i < 64 * P8; i += 128) {
        const int r = i / P8, c = i % P8 * 8;
        __nv_bfloat16* to = dst + r * LD + c;
        if (r < live && c < width)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(mt_addr(to)), "l"(src + (size_t)r * ld + c) : "memory");
        else
            *reinterpret_cast<uint4*>(to) = make_uint4(0u, 0u, 0u, 0u);
    }
}
__device__ __forceinline__ void mt_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void mt_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

__device__ __forceinline__ float2 mt_unpack(uint32_t v) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v));
}
// two 32-bit numbers as a pair of bfloat16 numbers and the pair of what is left
__device__ __forceinline__ void mt_split(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    const float2 h = mt_unpack(hi);
    lo = pack_bf16(a - h.x, b - h.y);
}

__global__ void __launch_bounds__(128) mlstm_tc_update_kernel(const MlstmTcArgs q) {
    __shared__ __align__(16) __nv_bfloat16 sk[64 * MT_LK], sv[64 * MT_LV];
    __shared__ float se[64];
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = q.c.p;
    const int d = p.d, dv = p.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, ch = blockIdx.z;
    const int tiles_v = (dv + 127) / 128;
    const int r0 = blockIdx.x / tiles_v * 64, v0 = blockIdx.x % tiles_v * 128;
    const int row0 = q.c.chunks[2 * ch], cnt = q.c.chunks[2 * ch + 1];
    const __nv_bfloat16* src = (const __nv_bfloat16*)p.x + (size_t)row0 * p.ldx;
    mt_stage<64, MT_LK>(sk, src + p.ck + h * d + r0, p.ldx, cnt, d - r0);
    mt_stage<128, MT_LV>(sv, src + p.cv + h * dv + v0, p.ldx, cnt, dv - v0);
    mt_commit();
    if (tid < 64) se[tid] = tid < cnt ? q.c.gates[3 * (size_t)p.H * q.c.T + (size_t)h * q.c.T + row0 + tid] : 0.f;
    float acc[16][4];
#pragma unroll
    for (int n = 0; n < 16; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    mt_wait();
    __syncthreads();
    const int g = lane >> 2, t2 = (lane & 3) * 2;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
        uint32_t a[4], hi[4], lo[4];      // keys of 16 tokens, transposed: rows are key channels
        ldmatrix_x4_trans(a, mt_addr(sk + (ks * 16 + (lane >> 4) * 8 + (lane & 7)) * MT_LK + 16 * warp + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int s = ks * 16 + (i >> 1) * 8 + t2;
            const float2 k = mt_unpack(a[i]);
            mt_split(k.x * se[s], k.y * se[s + 1], hi[i], lo[i]);
        }
#pragma unroll
        for (int n = 0; n < 16; n += 2) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, mt_addr(sv + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * MT_LV + 8 * (n + (lane >> 4))));
            mma_bf16_16816(acc[n], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
            mma_bf16_16816(acc[n], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
            mma_bf16_16816(acc[n + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
            mma_bf16_16816(acc[n + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
        }
    }
    float* U = q.U + ((size_t)ch * p.H + h) * d * dv;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = r0 + 16 * warp + g + 8 * half;
        if (r >= d) continue;
#pragma unroll
        for (int n = 0; n < 16; ++n) {
            const int c = v0 + 8 * n + t2;
            if (c < dv) *reinterpret_cast<float2*>(U + (size_t)r * dv + c) = make_float2(acc[n][2 * half], acc[n][2 * half + 1]);
        }
    }
    if (v0 == 0 && tid < 64 && r0 + tid < d) {
        float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int s = 0; s < 64; s += 4)
#pragma unroll
            for (int j = 0; j < 4; ++j) sum[j] = fmaf(se[s + j], __bfloat162float(sk[(s + j) * MT_LK + tid]), sum[j]);
        q.c.chunk_n[((size_t)ch * p.H + h) * d + r0 + tid] = (sum[0] + sum[1]) + (sum[2] + sum[3]);
    }
}

// grid (blocks of 256 items, heads, portions): an item is four numbers of S, or one of n behind them.
__global__ void __launch_bounds__(256) mlstm_tc_chain_kernel(const MlstmTcArgs q) {
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = q.c.p;
    const int h = blockIdx.y, size = p.d * p.dv, item = blockIdx.x * 256 + threadIdx.x;
    const int* po = q.c.portions + blockIdx.z * 4;
    const int cnt = po[1], slot = po[2], chunk0 = po[3], chunks = (cnt + ML_C - 1) / ML_C;
    const float* all = q.c.gates + 4 * (size_t)p.H * q.c.T + (size_t)h * q.c.T + po[0];    // at a chunk's last token
    auto last = [&](int i) { return all[min((i + 1) * ML_C, cnt) - 1]; };
    constexpr int AHEAD = 4;
    if (item * 4 < size) {
        float* state = p.S + ((size_t)slot * p.H + h) * size + item * 4;
        float S[4];
        load4(state, S);
        for (int i0 = 0; i0 < chunks; i0 += AHEAD) {
            float U[AHEAD][4], a[AHEAD];
#pragma unroll
            for (int u = 0; u < AHEAD; ++u)
                if (i0 + u < chunks) {
                    load4(q.U + ((size_t)(chunk0 + i0 + u) * p.H + h) * size + item * 4, U[u]);
                    a[u] = last(i0 + u);
                }
#pragma unroll
            for (int u = 0; u < AHEAD; ++u)
                if (i0 + u < chunks) {
                    __nv_bfloat16* to = q.S2 + ((size_t)(chunk0 + i0 + u) * p.H + h) * 2 * size + item * 4;
                    uint2 hi, lo;
                    mt_split(S[0], S[1], hi.x, lo.x);
                    mt_split(S[2], S[3], hi.y, lo.y);
                    *reinterpret_cast<uint2*>(to) = hi;
                    *reinterpret_cast<uint2*>(to + size) = lo;
#pragma unroll
                    for (int j = 0; j < 4; ++j) S[j] = fmaf(a[u], S[j], U[u][j]);
                }
        }
        store4(state, S);
    } else if (item - size / 4 < p.d) {
        const int r = item - size / 4;
        float* state = p.n + ((size_t)slot * p.H + h) * p.d + r;
        float n = *state;
        for (int i = 0; i < chunks; ++i) {
            float* at = q.c.chunk_n + ((size_t)(chunk0 + i) * p.H + h) * p.d + r;
            const float u = *at;
            *at = n;
            n = fmaf(last(i), n, u);
        }
        *state = n;
    }
}

constexpr size_t MT_OUT_SMEM = sizeof(float) * (64 * MT_LD + 4 * 64 + 128) + 2 * (2 * 64 * MT_LK + 2 * 64 * MT_LV);

template <typename TO>
__global__ void __launch_bounds__(128, 3) mlstm_tc_outputs_kernel(const MlstmTcArgs q) {
    extern __shared__ __align__(16) float smem[];
    float *sd = smem, *sa = sd + 64 * MT_LD, *sA = sa + 64, *sn = sA + 64, *sfloor = sn + 64, *sweight = sfloor + 64;
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(sweight + 128);
    __nv_bfloat16 *sk = sq + 64 * MT_LK, *sh = sk + 64 * MT_LK, *sl = sh + 64 * MT_LV;     // S: high part, rest
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = q.c.p;
    const int ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 128, tid = threadIdx.x, d = p.d, dv = p.dv;
    const int lane = tid & 31, warp = tid >> 5, g = lane >> 2, t2 = (lane & 3) * 2;
    const int row0 = q.c.chunks[2 * ch], cnt = q.c.chunks[2 * ch + 1];
    const size_t plane = (size_t)p.H * q.c.T;
    const float* ga = q.c.gates + (size_t)h * q.c.T + row0;
    const __nv_bfloat16* src = (const __nv_bfloat16*)p.x + (size_t)row0 * p.ldx;
    const __nv_bfloat16* S2 = q.S2 + ((size_t)ch * p.H + h) * 2 * d * dv;
    const float* nn = q.c.chunk_n + ((size_t)ch * p.H + h) * d;
    auto stage = [&](int k0) {
        mt_stage<64, MT_LK>(sq, src + p.cq + h * d + k0, p.ldx, cnt, d - k0);
        mt_stage<64, MT_LK>(sk, src + p.ck + h * d + k0, p.ldx, cnt, d - k0);
        mt_stage<128, MT_LV>(sh, S2 + (size_t)k0 * dv + v0, dv, d - k0, dv - v0);
        mt_stage<128, MT_LV>(sl, S2 + (size_t)d * dv + (size_t)k0 * dv + v0, dv, d - k0, dv - v0);
        mt_commit();
        if (tid < 64) sn[tid] = k0 + tid < d ? nn[k0 + tid] : 0.f;
    };
    stage(0);
    if (tid < 64) {
        sa[tid] = tid < cnt ? ga[tid] : 1.f;
    } else {
        const int t = tid - 64;
        sA[t] = t < cnt ? ga[4 * plane + t] : 0.f;
        sfloor[t] = t < cnt ? ga[2 * plane + t] : 1.f;
    }
    sweight[tid] = v0 + tid < dv ? p.w[h * dv + v0 + tid] : 0.f;
    __syncthreads();
    if (tid < 64) {          // b_s P(s, t) for W[t, s]
        float w = tid < cnt ? ga[plane + tid] : 0.f;
#pragma unroll 8
        for (int t = 0; t < 64; ++t) {
            if (t > tid) w *= sa[t];
            sd[t * MT_LD + tid] = t < tid ? 0.f : w;
        }
    }
    float o[16][4], w[8][4], qn[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < 16; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
#pragma unroll
    for (int n = 0; n < 8; ++n) w[n][0] = w[n][1] = w[n][2] = w[n][3] = 0.f;
    for (int k0 = 0; k0 < d; k0 += 64) {
        if (k0) {
            __syncthreads();                               // the last slab has been used
            stage(k0);
        }
        mt_wait();
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (k0 + kk * 16 >= d) break;
            uint32_t a[4];
            ldmatrix_x4(a, mt_addr(sq + (16 * warp + ((lane >> 3) & 1) * 8 + (lane & 7)) * MT_LK + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 v = mt_unpack(a[i]);
                const float* nr = sn + kk * 16 + (i >> 1) * 8 + t2;
                qn[i & 1] = fmaf(v.x, nr[0], fmaf(v.y, nr[1], qn[i & 1]));
            }
#pragma unroll
            for (int n = 0; n < 8; n += 2) {               // (tokens behind the warp's last row take no part)
                if (8 * n > 16 * warp + 15) break;
                uint32_t b[4];
                ldmatrix_x4(b, mt_addr(sk + (8 * n + (lane >> 4) * 8 + (lane & 7)) * MT_LK + kk * 16 + ((lane >> 3) & 1) * 8));
                mma_bf16_16816(w[n], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16_16816(w[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
#pragma unroll
            for (int n = 0; n < 16; n += 2) {
                const int at = (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * MT_LV + 8 * (n + (lane >> 4));
                uint32_t b[4], c[4];
                ldmatrix_x4_trans(b, mt_addr(sh + at));
                ldmatrix_x4_trans(c, mt_addr(sl + at));
                mma_bf16_16816(o[n], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16_16816(o[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                mma_bf16_16816(o[n], a[0], a[1], a[2], a[3], c[0], c[1]);
                mma_bf16_16816(o[n + 1], a[0], a[1], a[2], a[3], c[2], c[3]);
            }
        }
    }
    __syncthreads();
    mt_stage<128, MT_LV>(sh, src + p.cv + h * dv + v0, p.ldx, cnt, dv - v0);      // the values take the states' place,
    __nv_bfloat16* sg = sq;                                                        // the gate that of q and k
    if (!q.c.o) mt_stage<128, MT_LV>(sg, src + p.cg + h * dv + v0, p.ldx, cnt, dv - v0);
    mt_commit();
    const int tr[2] = {16 * warp + g, 16 * warp + g + 8};                          // this thread's two tokens
    float inv[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const float A = sA[tr[i]];
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            const float2 dec = *reinterpret_cast<const float2*>(sd + tr[i] * MT_LD + 8 * n + t2);
            w[n][2 * i] *= dec.x;
            w[n][2 * i + 1] *= dec.y;
            sum += w[n][2 * i] + w[n][2 * i + 1];
        }
        sum = fmaf(A, qn[i], sum);
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        // (q's scale multiplies both read-outs, here)
        inv[i] = p.q_scale / (fmaxf(fabsf(sum * p.q_scale), sfloor[tr[i]]) + 1e-6f);
#pragma unroll
        for (int n = 0; n < 16; ++n) {
            o[n][2 * i] *= A;
            o[n][2 * i + 1] *= A;
        }
    }
    mt_wait();
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
        if (ks > warp) break;
        uint32_t hi[4], lo[4];
        mt_split(w[2 * ks][0], w[2 * ks][1], hi[0], lo[0]);
        mt_split(w[2 * ks][2], w[2 * ks][3], hi[1], lo[1]);
        mt_split(w[2 * ks + 1][0], w[2 * ks + 1][1], hi[2], lo[2]);
        mt_split(w[2 * ks + 1][2], w[2 * ks + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int n = 0; n < 16; n += 2) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, mt_addr(sh + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * MT_LV + 8 * (n + (lane >> 4))));
            mma_bf16_16816(o[n], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
            mma_bf16_16816(o[n], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
            mma_bf16_16816(o[n + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
            mma_bf16_16816(o[n + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < 16; ++n) {                     // (columns beyond dv are zeros)
            o[n][2 * i] *= inv[i];
            o[n][2 * i + 1] *= inv[i];
            ss = fmaf(o[n][2 * i], o[n][2 * i], fmaf(o[n][2 * i + 1], o[n][2 * i + 1], ss));
        }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if (tr[i] >= cnt) continue;
        const size_t at = ((size_t)(row0 + tr[i]) * p.H + h) * dv;
        const float scale = 1.f / sqrtf(ss / (float)dv + p.eps);
        const __nv_bfloat16* gr = sg + tr[i] * MT_LV;
#pragma unroll
        for (int n = 0; n < 16; ++n) {
            const int c = 8 * n + t2;
            if (v0 + c >= dv) continue;
            if (q.c.o) {
                *reinterpret_cast<float2*>(q.c.o + at + v0 + c) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
                continue;
            }
            const float2 gate = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gr + c));
            const float2 wv = *reinterpret_cast<const float2*>(sweight + c);
            const float y0 = o[n][2 * i] * scale * wv.x / (1.f + expf(-gate.x));
            const float y1 = o[n][2 * i + 1] * scale * wv.y / (1.f + expf(-gate.y));
            TO* y = (TO*)p.y + at + v0 + c;
            if constexpr (sizeof(TO) == 2) *reinterpret_cast<__nv_bfloat162*>(y) = __floats2bfloat162_rn(y0, y1);
            else *reinterpret_cast<float2*>(y) = make_float2(y0, y1);
        }
    }
}

}  // namespace air

// As air_mlstm_portions (mlstm.cu) with x in bfloat16; d, dv, ldx and the columns of x multiples of 8.  Scratch: gates float32 [5, H, T], U float32
// [N, H, d, dv], S2 bfloat16 [N, H, 2, d, dv], chunk_n float32 [N, H, d], and o [T, H, dv] where dv > 128.
AIR_API int air_mlstm_portions_tc(const void* x, int ldx, int cq, int ck, int cv, int cg, const float* z, int ldz, int ci,
                                  int cf, const float* ib, const float* fb, const float* w, float* S, float* n, float* m,
                                  void* y, int out_dtype, const int* portions, int L, const int* chunks, int N,
                                  float* gates, float* U, void* S2, float* chunk_n, float* o, int T, int H, int d, int dv,
                                  float cap, float q_scale, float eps, cudaStream_t stream) {
    if (L <= 0 || N <= 0) return 0;
    const int v_blocks = (dv + 127) / 128, d_blocks = (d + 63) / 64;
    if (H <= 0 || H > 65535 || d <= 0 || dv <= 0 || L > 65535 || N > 65535 || v_blocks > 65535 || !(cap > 0.f) || !gates || !U ||
        !S2 || !chunk_n || (v_blocks > 1 && !o) || ((ldx | cq | ck | cv | cg | d | dv) & 7) ||
        (((uintptr_t)x | (uintptr_t)U | (uintptr_t)S2 | (uintptr_t)S | (uintptr_t)y) & 15))
        return AIR_ERR_BAD_ARGUMENT;
    air::MlstmTcArgs q;
    q.c.p = air::MlstmArgs{x, ldx, z, ldz, cq, ck, cv, cg, ci, cf, ib, fb, w, S, n, m, y, nullptr, nullptr, H, d, dv, cap, q_scale, eps};
    q.c.portions = portions; q.c.chunks = chunks; q.c.gates = gates; q.c.chunk_S = nullptr; q.c.chunk_n = chunk_n;
    q.c.o = v_blocks > 1 ? o : nullptr; q.c.T = T; q.c.vec = 1;
    q.U = U; q.S2 = (__nv_bfloat16*)S2;
    int rc = air::launch_mlstm_gates(q.c, L, stream);
    if (rc) return rc;
    rc = air::launch(air::mlstm_tc_update_kernel, dim3(d_blocks * v_blocks, H, N), 128, 0, stream, q);
    if (rc) return rc;
    rc = air::launch(air::mlstm_tc_chain_kernel, dim3((d * dv / 4 + d + 255) / 256, H, L), 256, 0, stream, q);
    if (rc) return rc;
    AIR_DISPATCH(out_dtype, TO, {
        auto kernel = air::mlstm_tc_outputs_kernel<TO>;
        cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)air::MT_OUT_SMEM);
        if (err != cudaSuccess) return (int)err;
        rc = air::launch(kernel, dim3(N, H, v_blocks), 128, air::MT_OUT_SMEM, stream, q);
        if (rc || v_blocks == 1) return rc;
        return air::launch(air::mlstm_finish_kernel<__nv_bfloat16, TO>, dim3(N, H), 128, 0, stream, q.c);
    });
    return 0;
}

AIR_API int air_trace_set_mlstm_tc(unsigned long long* buffer) { return air::set_trace_here(buffer); }
