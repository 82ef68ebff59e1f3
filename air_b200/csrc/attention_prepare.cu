// What stands between the fused projection of an attention layer and its attention kernel, for layers whose
// keys and values differ in size or that want more than a bias and a rotation:
//
//   proj [T, ld] float32 holds, per token, q (H heads of dk), k (G heads of dk), v (G heads of dv) and, where the
//   layer gates its heads, H gate logits, in this order.  Per token: add the bias; rotate the first `rot` elements
//   of every head of q and k (element i with i + rot/2, angle position * inv_freq[i], evaluated here in 32-bit);
//   mix the values with those of an earlier layer, v = (1 - lambda) v + lambda v_first (v_mode 2), or hand them on
//   as v_first (v_mode 1); write q to q_out [T, H, dk], k and v into the token's place in the pages, and
//   sigmoid(gate logits) to gate_out [T, H].
//
// A page holds the keys [G, P, dk] and behind them the values [G, P, dv]; with dk == dv that is [2, G, P, d], the
// layout of the other attention kernels.
#include "common.cuh"

namespace air {

template <typename TO>
__global__ void __launch_bounds__(1024)
qkv_prepare_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ bias,
                   const float* __restrict__ inv_freq, int rot, const int* __restrict__ positions,
                   const int* __restrict__ token_seq, const int* __restrict__ block_table, int max_blocks,
                   TO* __restrict__ q_out, TO* __restrict__ cache, float* __restrict__ gate_out,
                   float* __restrict__ v_first, int v_mode, const float* __restrict__ lambda,
                   int H, int G, int dk, int dv, int P, int* status) {
    pdl_enter(TR_QKV_PREPARE);
    const int t = blockIdx.x;
    const int slot = token_seq[t];
    if (slot < 0) return;
    const int pos = positions[t];
    const float* in = proj + (size_t)t * ld;
    const int half = rot / 2;
    const int page = block_table[(size_t)slot * max_blocks + pos / P];
    TO* kdst = nullptr;
    TO* vdst = nullptr;
    if (page < 0) {
        if (threadIdx.x == 0 && status) atomicExch(status, 2);
    } else {
        TO* base = cache + (size_t)page * G * P * (dk + dv);
        kdst = base + (size_t)(pos % P) * dk;
        vdst = base + (size_t)G * P * dk + (size_t)(pos % P) * dv;
    }
    // q and k: one item per pair of rotated elements and per element behind the rotated part
    const int per_head = dk - half;
    for (int idx = threadIdx.x; idx < (H + G) * per_head; idx += blockDim.x) {
        const int head = idx / per_head, j = idx % per_head;
        const int col = head * dk;
        const int i0 = j < half ? j : j + half;
        float a = in[col + i0] + (bias ? bias[col + i0] : 0.f), b = 0.f;
        if (j < half) {
            b = in[col + i0 + half] + (bias ? bias[col + i0 + half] : 0.f);
            float s, c;
            sincosf((float)pos * inv_freq[j], &s, &c);
            const float ra = a * c - b * s, rb = b * c + a * s;
            a = ra;
            b = rb;
        }
        TO* dst = head < H ? q_out + ((size_t)t * H + head) * dk
                           : (kdst ? kdst + (size_t)(head - H) * P * dk : nullptr);
        if (dst) {
            dst[i0] = from_float<TO>(a);
            if (j < half) dst[i0 + half] = from_float<TO>(b);
        }
    }
    const int vcol = (H + G) * dk;
    const float lam = v_mode == 2 ? lambda[0] : 0.f;
    for (int idx = threadIdx.x; idx < G * dv; idx += blockDim.x) {
        float v = in[vcol + idx] + (bias ? bias[vcol + idx] : 0.f);
        if (v_mode == 1) v_first[(size_t)t * G * dv + idx] = v;
        else if (v_mode == 2) v = (1.f - lam) * v + lam * v_first[(size_t)t * G * dv + idx];
        if (vdst) vdst[(size_t)(idx / dv) * P * dv + idx % dv] = from_float<TO>(v);
    }
    if (gate_out) {
        const int gcol = vcol + G * dv;
        for (int h = threadIdx.x; h < H; h += blockDim.x) {
            const float z = in[gcol + h] + (bias ? bias[gcol + h] : 0.f);
            gate_out[(size_t)t * H + h] = 1.f / (1.f + expf(-z));
        }
    }
}

}  // namespace air

AIR_API int air_qkv_prepare(const float* proj, int ld, const float* bias, const float* inv_freq, int rot,
                            const int* positions, const int* token_seq, const int* block_table, int max_blocks,
                            void* q_out, void* cache, int out_dtype, float* gate_out, float* v_first, int v_mode,
                            const float* lambda, int T, int H, int G, int dk, int dv, int P, int* status,
                            cudaStream_t stream) {
    if (T <= 0) return 0;
    if (rot < 0 || rot > dk || (rot & 1) || (rot > 0 && !inv_freq) || v_mode < 0 || v_mode > 2 ||
        (v_mode && !v_first) || (v_mode == 2 && !lambda))
        return AIR_ERR_BAD_ARGUMENT;
    AIR_DISPATCH(out_dtype, TO, return air::launch(air::qkv_prepare_kernel<TO>, T, T <= 64 ? 1024 : 256, 0, stream, proj, ld, bias,
                                                   inv_freq, rot, positions, token_seq, block_table, max_blocks,
                                                   (TO*)q_out, (TO*)cache, gate_out, v_first, v_mode, lambda, H, G, dk,
                                                   dv, P, status));
    return 0;
}

AIR_API int air_trace_set_attention_prepare(unsigned long long* buffer) { return air::set_trace_here(buffer); }

// The same step for layers that normalise queries and keys per head before they rotate them, and whose rotation may
// pair neighbours:
//
//   q and k heads: x <- x / sqrt(mean(x^2) + eps) * w (w [dk], one for all heads of q, one for all heads of k; absent:
//   no norm); then the first `rot` elements are rotated, pair j by the angle position * freq[j], where pair j is
//   (2j, 2j + 1) (pairing 1) or (j, j + rot/2) (pairing 0); cos and sin are multiplied by `magnitude`.  The angle is
//   the product of the position and a 64-bit frequency, taken in 64-bit (cos_sin_of), once per token.
//   v is copied.  Pages as above.  A bias (float32 [(H + G) dk + G dv]) is added to q, k and v first.  With `whole`
//   the norm is taken over ALL heads of q at once (and all heads of k): x / sqrt(mean over H dk (x^2) + eps) * w with
//   w of that whole size (q_w [H dk], k_w [G dk]).
//
//   q_scale [H] multiplies the heads of q behind norm and rotation (a factor per head on the scores).  v_freq [v_rot / 2]
//   rotates the first v_rot elements of every head of v as well, in the same pairing, before it is written (no magnitude).
//   Without write_kv proj holds q alone and nothing is written to the pages (a layer that reads another layer's keys).
//
// One block per token, one warp per head of q or k; a lane holds up to QKN_PAIRS pairs of its head.  Without any rotation
// and with a norm per head or none (qk_normed_rows_kernel) nothing pairs up: a lane holds four neighbours, as many lanes as a
// head needs (a power of two) take it, and the heads of a token are spread over the blocks of a row of the grid.
//
// turn_heads_kernel  rotates the first `rot` elements of every head of x [T, H, n] by sign * position * freq[j], in place:
//                    values that were rotated by their own positions and summed over positions are turned back by the
//                    query's.
namespace air {

constexpr int QKN_PAIRS = 4;      // head sizes up to 64 * QKN_PAIRS

template <typename TO>
__global__ void __launch_bounds__(256)
qk_normed_prepare_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ q_w,
                         const float* __restrict__ k_w, float eps, const double* __restrict__ freq, int rot,
                         int pairing, float magnitude, const int* __restrict__ positions,
                         const int* __restrict__ token_seq, const int* __restrict__ block_table, int max_blocks,
                         TO* __restrict__ q_out, TO* __restrict__ cache, int H, int G, int dk, int dv, int P,
                         int* status, const float* __restrict__ bias, int whole, const float* __restrict__ q_scale,
                         const double* __restrict__ v_freq, int v_rot, int write_kv) {
    __shared__ float cs[128], sn[128], vcs[128], vsn[128], scratch[32];
    pdl_enter(TR_QK_NORMED_PREPARE);
    const int t = blockIdx.x;
    const int slot = token_seq[t];
    if (slot < 0) return;
    const int pos = positions[t];
    const float* in = proj + (size_t)t * ld;
    const int half = rot / 2;
    for (int j = threadIdx.x; j < half; j += blockDim.x) {
        float s, c;
        cos_sin_of((double)pos, freq[j], c, s);
        cs[j] = c * magnitude;
        sn[j] = s * magnitude;
    }
    const int vhalf = v_rot / 2;
    if (write_kv)
        for (int j = threadIdx.x; j < vhalf; j += blockDim.x) cos_sin_of((double)pos, v_freq[j], vcs[j], vsn[j]);
    TO* kdst = nullptr;
    TO* vdst = nullptr;
    if (write_kv) {
        const int page = block_table[(size_t)slot * max_blocks + pos / P];
        if (page < 0) {
            if (threadIdx.x == 0 && status) atomicExch(status, 2);
        } else {
            TO* base = cache + (size_t)page * G * P * (dk + dv);
            kdst = base + (size_t)(pos % P) * dk;
            vdst = base + (size_t)G * P * dk + (size_t)(pos % P) * dv;
        }
    }
    const int heads = write_kv ? H + G : H;
    __syncthreads();
    float whole_q = 1.f, whole_k = 1.f;
    if (whole && q_w) {      // one scale for all heads of q and one for all heads of k
        // (four loads of a thread under way at once: the sums are a chain of latencies otherwise)
        float sq = 0.f, sk = 0.f;
        const int n = heads * dk, step = blockDim.x;
        for (int i0 = threadIdx.x; i0 < n; i0 += 4 * step) {
            float v[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int i = i0 + u * step;
                v[u] = i < n ? in[i] + (bias ? bias[i] : 0.f) : 0.f;
            }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                if (i0 + u * step < H * dk) sq = fmaf(v[u], v[u], sq);
                else sk = fmaf(v[u], v[u], sk);
            }
        }
        whole_q = 1.f / sqrtf(block_sum(sq, scratch) / (float)(H * dk) + eps);
        whole_k = 1.f / sqrtf(block_sum(sk, scratch) / (float)(G * dk) + eps);
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int pairs = dk / 2;
    for (int head = warp; head < heads; head += warps) {
        const float* x = in + (size_t)head * dk;
        const float* hb = bias ? bias + (size_t)head * dk : nullptr;
        const float* w = head < H ? q_w : k_w;
        if (w && whole) w += (size_t)(head < H ? head : head - H) * dk;
        float a[QKN_PAIRS], b[QKN_PAIRS];
        int ia[QKN_PAIRS], ib[QKN_PAIRS];
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < QKN_PAIRS; ++c) {
            const int j = lane + 32 * c;
            a[c] = b[c] = 0.f;
            ia[c] = ib[c] = 0;
            if (j < pairs) {
                ia[c] = (pairing == 0 && j < half) ? j : 2 * j;
                ib[c] = (pairing == 0 && j < half) ? j + half : 2 * j + 1;
                a[c] = x[ia[c]] + (hb ? hb[ia[c]] : 0.f);
                b[c] = x[ib[c]] + (hb ? hb[ib[c]] : 0.f);
                ss += a[c] * a[c] + b[c] * b[c];
            }
        }
        ss = warp_sum(ss);
        const float scale = !w ? 1.f : whole ? (head < H ? whole_q : whole_k) : 1.f / sqrtf(ss / (float)dk + eps);
        TO* dst = head < H ? q_out + ((size_t)t * H + head) * dk
                           : (kdst ? kdst + (size_t)(head - H) * P * dk : nullptr);
#pragma unroll
        for (int c = 0; c < QKN_PAIRS; ++c) {
            const int j = lane + 32 * c;
            if (j >= pairs) continue;
            float u = a[c], v = b[c];
            if (w) {
                u = u * scale * w[ia[c]];
                v = v * scale * w[ib[c]];
            }
            if (j < half) {
                const float ru = u * cs[j] - v * sn[j], rv = v * cs[j] + u * sn[j];
                u = ru;
                v = rv;
            }
            if (q_scale && head < H) {
                u *= q_scale[head];
                v *= q_scale[head];
            }
            if (dst) {
                dst[ia[c]] = from_float<TO>(u);
                dst[ib[c]] = from_float<TO>(v);
            }
        }
    }
    const int vcol = (H + G) * dk;
    if (!vdst) return;
    // v: one item per pair of rotated elements and per element behind them
    const int per_head = dv - vhalf;
    for (int idx = threadIdx.x; idx < G * per_head; idx += blockDim.x) {
        const int g = idx / per_head, j = idx % per_head;
        const int i0 = j >= vhalf ? j + vhalf : pairing == 0 ? j : 2 * j, i1 = pairing == 0 ? i0 + vhalf : i0 + 1;
        const int col = vcol + g * dv;
        TO* dst = vdst + (size_t)g * P * dv;
        const float a = in[col + i0] + (bias ? bias[col + i0] : 0.f);
        if (j >= vhalf) {
            dst[i0] = from_float<TO>(a);
            continue;
        }
        const float b = in[col + i1] + (bias ? bias[col + i1] : 0.f);
        dst[i0] = from_float<TO>(a * vcs[j] - b * vsn[j]);
        dst[i1] = from_float<TO>(b * vcs[j] + a * vsn[j]);
    }
}

template <typename TO>
__global__ void __launch_bounds__(256)
qk_normed_rows_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ q_w, const float* __restrict__ k_w,
                      float eps, const int* __restrict__ positions, const int* __restrict__ token_seq,
                      const int* __restrict__ block_table, int max_blocks, TO* __restrict__ q_out, TO* __restrict__ cache,
                      int H, int G, int dk, int dv, int P, int* status, const float* __restrict__ bias,
                      const float* __restrict__ q_scale, int write_kv, int lanes) {
    pdl_enter(TR_QK_NORMED_PREPARE);
    const int t = blockIdx.x;
    const int slot = token_seq[t];
    if (slot < 0) return;
    const int pos = positions[t];
    const float* in = proj + (size_t)t * ld;
    TO* kdst = nullptr;
    TO* vdst = nullptr;
    if (write_kv) {
        const int page = block_table[(size_t)slot * max_blocks + pos / P];
        if (page < 0) {
            if (threadIdx.x == 0 && status) atomicExch(status, 2);
        } else {
            TO* base = cache + (size_t)page * G * P * (dk + dv);
            kdst = base + (size_t)(pos % P) * dk;
            vdst = base + (size_t)G * P * dk + (size_t)(pos % P) * dv;
        }
    }
    const int heads = write_kv ? H + G : H;
    const int head = blockIdx.y * (256 / lanes) + threadIdx.x / lanes, l = threadIdx.x % lanes;
    const bool live = head < heads;
    constexpr int M = QKN_PAIRS / 2;      // pieces of four per lane
    float x[M][4], ss = 0.f;
#pragma unroll
    for (int c = 0; c < M; ++c) {
        const int i = (l + c * lanes) * 4;
        if (live && i < dk) {
            load4(in + (size_t)head * dk + i, x[c]);
            if (bias) {
                float b[4];
                load4(bias + (size_t)head * dk + i, b);
#pragma unroll
                for (int j = 0; j < 4; ++j) x[c][j] += b[j];
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) ss = fmaf(x[c][j], x[c][j], ss);
        }
    }
    for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (live) {
        const float* w = head < H ? q_w : k_w;
        const float scale = (w ? 1.f / sqrtf(ss / (float)dk + eps) : 1.f), more = q_scale && head < H ? q_scale[head] : 1.f;
        TO* dst = head < H ? q_out + ((size_t)t * H + head) * dk : (kdst ? kdst + (size_t)(head - H) * P * dk : nullptr);
#pragma unroll
        for (int c = 0; c < M; ++c) {
            const int i = (l + c * lanes) * 4;
            if (i >= dk || !dst) continue;
            float wv[4] = {1.f, 1.f, 1.f, 1.f};
            if (w) load4(w + i, wv);
#pragma unroll
            for (int j = 0; j < 4; ++j) x[c][j] = x[c][j] * scale * wv[j] * more;
            store4(dst + i, x[c]);
        }
    }
    if (!vdst) return;
    const int vcol = (H + G) * dk;
    for (int i = (blockIdx.y * 256 + threadIdx.x) * 4; i < G * dv; i += gridDim.y * 1024) {
        float v[4];
        load4(in + vcol + i, v);
        if (bias) {
            float b[4];
            load4(bias + vcol + i, b);
#pragma unroll
            for (int j = 0; j < 4; ++j) v[j] += b[j];
        }
        store4(vdst + (size_t)(i / dv) * P * dv + i % dv, v);
    }
}

template <typename TX>
__global__ void __launch_bounds__(256)
turn_heads_kernel(TX* __restrict__ x, const double* __restrict__ freq, int rot, int pairing, double sign,
                  const int* __restrict__ positions, const int* __restrict__ token_seq, int H, int n) {
    __shared__ float cs[128], sn[128];
    pdl_enter(TR_TURN);
    const int t = blockIdx.x;
    if (token_seq[t] < 0) return;
    const int half = rot / 2;
    for (int j = threadIdx.x; j < half; j += blockDim.x)
        cos_sin_of(sign * (double)positions[t], freq[j], cs[j], sn[j]);
    __syncthreads();
    for (int idx = threadIdx.x; idx < H * half; idx += blockDim.x) {
        const int h = idx / half, j = idx % half;
        TX* row = x + ((size_t)t * H + h) * n;
        const int i0 = pairing == 0 ? j : 2 * j, i1 = pairing == 0 ? j + half : 2 * j + 1;
        const float a = to_float(row[i0]), b = to_float(row[i1]);
        row[i0] = from_float<TX>(a * cs[j] - b * sn[j]);
        row[i1] = from_float<TX>(b * cs[j] + a * sn[j]);
    }
}

}  // namespace air

AIR_API int air_qk_normed_prepare(const float* proj, int ld, const float* q_w, const float* k_w, float eps,
                                  const double* freq, int rot, int pairing, float magnitude, const int* positions,
                                  const int* token_seq, const int* block_table, int max_blocks, void* q_out,
                                  void* cache, int out_dtype, int T, int H, int G, int dk, int dv, int P, int* status,
                                  const float* bias, int whole, const float* q_scale, const double* v_freq, int v_rot,
                                  int write_kv, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (v_rot < 0 || v_rot > dv || (v_rot & 1) || v_rot > 256 || (v_rot > 0 && !v_freq)) return AIR_ERR_BAD_ARGUMENT;
    if (rot < 0 || rot > dk || (rot & 1) || (dk & 1) || rot > 256 || dk > 64 * air::QKN_PAIRS || (rot > 0 && !freq) ||
        pairing < 0 || pairing > 1 || (write_kv && (!q_w) != (!k_w)))
        return AIR_ERR_BAD_ARGUMENT;
    auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    if (rot == 0 && v_rot == 0 && !whole && dk % 4 == 0 && (!write_kv || dv % 4 == 0) && ld % 4 == 0 && al(proj) && al(q_w) &&
        al(k_w) && al(q_out) && al(cache) && al(bias)) {
        int lanes = 1;
        while (lanes < 32 && lanes * 4 < dk) lanes *= 2;
        const int heads = write_kv ? H + G : H, per_block = 256 / lanes;
        const dim3 grid(T, (heads + per_block - 1) / per_block);
        AIR_DISPATCH(out_dtype, TO, return air::launch(air::qk_normed_rows_kernel<TO>, grid, 256, 0, stream, proj, ld, q_w, k_w,
                                                       eps, positions, token_seq, block_table, max_blocks, (TO*)q_out,
                                                       (TO*)cache, H, G, dk, dv, P, status, bias, q_scale, write_kv, lanes));
    }
    AIR_DISPATCH(out_dtype, TO, return air::launch(air::qk_normed_prepare_kernel<TO>, T, 256, 0, stream, proj, ld, q_w,
                                                   k_w, eps, freq, rot, pairing, magnitude, positions, token_seq,
                                                   block_table, max_blocks, (TO*)q_out, (TO*)cache, H, G, dk, dv, P,
                                                   status, bias, whole, q_scale, v_freq, v_rot, write_kv));
    return 0;
}

AIR_API int air_turn_heads(void* x, int dtype, const double* freq, int rot, int pairing, int back, const int* positions,
                           const int* token_seq, int T, int H, int n, cudaStream_t stream) {
    if (T <= 0 || rot == 0) return 0;
    if (rot < 0 || rot > n || (rot & 1) || rot > 256 || !freq || pairing < 0 || pairing > 1) return AIR_ERR_BAD_ARGUMENT;
    AIR_DISPATCH(dtype, TX, return air::launch(air::turn_heads_kernel<TX>, T, 256, 0, stream, (TX*)x, freq, rot, pairing,
                                               back ? -1.0 : 1.0, positions, token_seq, H, n));
    return 0;
}
