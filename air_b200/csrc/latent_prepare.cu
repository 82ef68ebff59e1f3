// What stands between the first projection of a latent-attention layer and its attention kernel.
//
//   q [T, ldq] float32 holds, per token, H heads of [d plain | rot rotated] and, where the layer makes its own latent
//   (owns), c [T, ldc] the latent (R columns) and behind it one rotated key part kr (rot columns) for all heads; the
//   two may be bands of columns of one product.
//   Per token: c <- c / sqrt(mean(c^2) + eps) * w_c; kr and the rotated part of every head of q are turned, pair i by
//   the angle position * freq[i] (a 64-bit product, cos and sin taken in 64-bit once per token), where pair i is
//   (i, i + rot/2) (pairing 0) or (2i, 2i + 1) (pairing 1);
//   the row [c | kr] goes to the token's place in the pages ([P, R + rot] per page, no heads); the plain part of q goes
//   to q_plain [T, H, d] (the matrix product that absorbs the key expansion reads it), the rotated part to
//   q_full[t, h, R : R + rot] (float32; that product fills q_full[t, h, 0 : R]).  rot may be 0 (no rotated parts).
//   Where the layer gates its heads, gate [T, ldg] holds one logit per head, and gate_out[t, h] = sigmoid(logit)
//   (float32).
//
// One block per token.
//
// band_rmsnorm_kernel: rows of a band of columns over their root mean square, out = x / sqrt(mean(x^2) + eps) * w (a
//   query's latent on its way to the product that makes the heads), zeros behind them up to out's width ldo.  One block
//   per row.
#include "common.cuh"

namespace air {

template <typename TO>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(const float* __restrict__ q_in, int ldq, const float* __restrict__ c_in, int ldc,
                      const float* __restrict__ gate_in, int ldg, const float* __restrict__ c_w, float eps, int pairing,
                      const double* __restrict__ freq, const int* __restrict__ positions,
                      const int* __restrict__ token_seq, const int* __restrict__ block_table, int max_blocks,
                      TO* __restrict__ q_plain, float* __restrict__ q_full, TO* __restrict__ cache, int owns, int H,
                      int d, int rot, int R, int P, float* __restrict__ gate_out, int* status, int vec_q, int vec_c) {
    __shared__ float cs[128], sn[128];
    __shared__ float scratch[32];
    pdl_enter(TR_LATENT_PREPARE);
    const int t = blockIdx.x;
    const int slot = token_seq[t];
    if (slot < 0) return;
    const int pos = positions[t];
    const float* in = q_in + (size_t)t * ldq;
    const int half = rot / 2;
    for (int j = threadIdx.x; j < half; j += blockDim.x) {
        double s, c;
        sincos((double)pos * freq[j], &s, &c);
        cs[j] = (float)c;
        sn[j] = (float)s;
    }
    __syncthreads();
    const int qw = d + rot;
    if (vec_q) {         // four numbers of a head at a time (d, rot and ldq multiples of 4, 16-byte boundaries)
        for (int idx = threadIdx.x * 4; idx < H * d; idx += blockDim.x * 4) {
            const int h = idx / d, i = idx % d;
            float x[4];
            load4(in + h * qw + i, x);
            store4(q_plain + ((size_t)t * H + h) * d + i, x);
        }
    } else {
        for (int idx = threadIdx.x; idx < H * d; idx += blockDim.x) {
            const int h = idx / d, i = idx % d;
            q_plain[((size_t)t * H + h) * d + i] = from_float<TO>(in[h * qw + i]);
        }
    }
    for (int idx = threadIdx.x; idx < H * half; idx += blockDim.x) {
        const int h = idx / half, j = idx % half;
        const int i0 = pairing ? 2 * j : j, i1 = pairing ? i0 + 1 : j + half;
        const float u = in[h * qw + d + i0], v = in[h * qw + d + i1];
        float* dst = q_full + ((size_t)t * H + h) * (R + rot) + R;
        dst[i0] = u * cs[j] - v * sn[j];
        dst[i1] = v * cs[j] + u * sn[j];
    }
    if (gate_out)
        for (int h = threadIdx.x; h < H; h += blockDim.x)
            gate_out[(size_t)t * H + h] = 1.f / (1.f + expf(-gate_in[(size_t)t * ldg + h]));
    if (!owns) return;
    const int page = block_table[(size_t)slot * max_blocks + pos / P];
    if (page < 0) {
        if (threadIdx.x == 0 && status) atomicExch(status, 2);
        return;
    }
    TO* row = cache + ((size_t)page * P + pos % P) * (R + rot);
    const float* c = c_in + (size_t)t * ldc;
    float ss = 0.f;
    if (vec_c) {
        for (int i = threadIdx.x * 4; i < R; i += blockDim.x * 4) {
            float x[4];
            load4(c + i, x);
#pragma unroll
            for (int j = 0; j < 4; ++j) ss += x[j] * x[j];
        }
    } else {
        for (int i = threadIdx.x; i < R; i += blockDim.x) ss += c[i] * c[i];
    }
    const float total = block_sum(ss, scratch);
    const float scale = 1.f / sqrtf(total / (float)R + eps);
    if (vec_c) {
        for (int i = threadIdx.x * 4; i < R; i += blockDim.x * 4) {
            float x[4], wv[4];
            load4(c + i, x);
            load4(c_w + i, wv);
#pragma unroll
            for (int j = 0; j < 4; ++j) x[j] = x[j] * scale * wv[j];
            store4(row + i, x);
        }
    } else {
        for (int i = threadIdx.x; i < R; i += blockDim.x) row[i] = from_float<TO>(c[i] * scale * c_w[i]);
    }
    for (int j = threadIdx.x; j < half; j += blockDim.x) {
        const int i0 = R + (pairing ? 2 * j : j), i1 = pairing ? i0 + 1 : i0 + half;
        const float u = c[i0], v = c[i1];
        row[i0] = from_float<TO>(u * cs[j] - v * sn[j]);
        row[i1] = from_float<TO>(v * cs[j] + u * sn[j]);
    }
}

template <typename TO>
__global__ void __launch_bounds__(256)
band_rmsnorm_kernel(const float* __restrict__ x, int ld, const float* __restrict__ w, float eps, TO* __restrict__ out, int ldo,
                    int n, int vec) {
    __shared__ float scratch[32];
    pdl_enter(TR_LATENT_PREPARE);
    const float* row = x + (size_t)blockIdx.x * ld;
    TO* dst = out + (size_t)blockIdx.x * ldo;
    float ss = 0.f;
    if (vec) {
        for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
            float v[4];
            load4(row + i, v);
#pragma unroll
            for (int j = 0; j < 4; ++j) ss = fmaf(v[j], v[j], ss);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(row[i], row[i], ss);
    }
    const float scale = 1.f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
    if (vec) {
        for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
            float v[4], wv[4];
            load4(row + i, v);
            load4(w + i, wv);
#pragma unroll
            for (int j = 0; j < 4; ++j) v[j] = v[j] * scale * wv[j];
            store4(dst + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) dst[i] = from_float<TO>(row[i] * scale * w[i]);
    }
    for (int i = n + threadIdx.x; i < ldo; i += blockDim.x) dst[i] = from_float<TO>(0.f);
}

}  // namespace air

AIR_API int air_latent_prepare(const float* q, int ldq, const float* c, int ldc, const float* gate, int ldg, const float* c_w,
                               float eps, const double* freq, int pairing, const int* positions, const int* token_seq,
                               const int* block_table, int max_blocks, void* q_plain, float* q_full, void* cache,
                               int out_dtype, int owns, int T, int H, int d, int rot, int R, int P, float* gate_out,
                               int* status, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (rot < 0 || (rot & 1) || rot > 256 || (rot > 0 && !freq) || (owns && (!c_w || !c || ldc < R + rot)) || d <= 0 || R <= 0 ||
        ldq < H * (d + rot) || (gate_out && (!gate || ldg < H)) || pairing < 0 || pairing > 1)
        return AIR_ERR_BAD_ARGUMENT;
    const int vec_q = d % 4 == 0 && rot % 4 == 0 && ldq % 4 == 0 && (((uintptr_t)q | (uintptr_t)q_plain) & 15) == 0;
    const int vec_c = R % 4 == 0 && rot % 4 == 0 && ldc % 4 == 0 && (((uintptr_t)c | (uintptr_t)c_w | (uintptr_t)cache) & 15) == 0;
    AIR_DISPATCH(out_dtype, TO, return air::launch(air::latent_prepare_kernel<TO>, T, 256, 0, stream, q, ldq, c, ldc, gate,
                                                   ldg, c_w, eps, pairing, freq, positions, token_seq, block_table,
                                                   max_blocks, (TO*)q_plain, q_full, (TO*)cache, owns, H, d, rot, R, P,
                                                   gate_out, status, vec_q, vec_c));
    return 0;
}

// x [T, ld] float32 (the first n columns), w float32 [n], out [T, ldo].
AIR_API int air_band_rmsnorm(const float* x, int ld, const float* w, float eps, void* out, int out_dtype, int ldo, int T, int n,
                             cudaStream_t stream) {
    if (T <= 0) return 0;
    if (n <= 0 || ld < n || ldo < n) return AIR_ERR_BAD_ARGUMENT;
    const int vec = n % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
    int threads = ((vec ? n / 4 : n) + 31) / 32 * 32;
    if (threads > 256) threads = 256;
    AIR_DISPATCH(out_dtype, TO, return air::launch(air::band_rmsnorm_kernel<TO>, T, threads, 0, stream, x, ld, w, eps, (TO*)out,
                                                   ldo, n, vec));
    return 0;
}

AIR_API int air_trace_set_latent_prepare(unsigned long long* buffer) { return air::set_trace_here(buffer); }
