// What the kernels of mLSTM's matrix memory share (mlstm.cu says what is computed, and how portions are cut into chunks).
#pragma once

#include "common.cuh"

namespace air {

constexpr int ML_THREADS = 256;

struct MlstmArgs {
    const void* x; int ldx;            // [T, ldx], float32 or bfloat16: q, k, v, g start at columns cq, ck, cv, cg
    const float* z; int ldz;           // [T, ldz]: the gates' logits start at columns ci, cf
    int cq, ck, cv, cg, ci, cf;
    const float* ib; const float* fb;  // [H]
    const float* w;                    // [H * dv]
    float* S; float* n; float* m;
    void* y;                           // [T, H * dv]
    const int* q_start; const int* slots;
    int H, d, dv;
    float cap, q_scale, eps;
};

constexpr int ML_C = 64;                   // tokens of a chunk

struct MlstmChunkArgs {
    MlstmArgs p;
    const int* portions;                   // [L, 4]: first row, tokens, slot, first chunk
    const int* chunks;                     // [N, 2]: first row, tokens
    float* gates;                          // [5, H, T]: a, b, exp(-m), b P(t, end) and A of every token in its chunk
    float* chunk_S; float* chunk_n;        // [N, H, d, dv], [N, H, d]: the states ahead of every chunk
    float* o;                              // [T, H, dv] read-outs where a head's v takes several blocks, else null
    int T, vec;                            // vec: x's rows and columns allow 16-byte accesses
};

int launch_mlstm_gates(const MlstmChunkArgs& c, int L, cudaStream_t stream);     // mlstm.cu

// One warp per (token of a portion, head): the norm, the weight and the gate of read-outs that several blocks have written.
template <typename TX, typename TO>
__global__ void __launch_bounds__(128) mlstm_finish_kernel(const MlstmChunkArgs c) {
    pdl_enter(TR_MLSTM);
    const MlstmArgs& p = c.p;
    const int row0 = c.chunks[2 * blockIdx.x], cnt = c.chunks[2 * blockIdx.x + 1], h = blockIdx.y, lane = threadIdx.x & 31;
    for (int t = threadIdx.x >> 5; t < cnt; t += 4) {
        const size_t at = ((size_t)(row0 + t) * p.H + h) * p.dv;
        float ss = 0.f;
        for (int i = lane; i < p.dv; i += 32) ss = fmaf(c.o[at + i], c.o[at + i], ss);
        const float scale = 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
        const TX* gr = (const TX*)p.x + (size_t)(row0 + t) * p.ldx + p.cg + h * p.dv;
        for (int i = lane; i < p.dv; i += 32)
            ((TO*)p.y)[at + i] = from_float<TO>(c.o[at + i] * scale * p.w[h * p.dv + i] / (1.f + expf(-to_float(gr[i]))));
    }
}

}  // namespace air
