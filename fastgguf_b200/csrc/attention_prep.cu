// What stands between an attention mixer's projections and its attention kernel when the mixer does more than rotate:
//
//   * fg_qkv_prepare: per token row, on the float32 projections q | k | v of a step - add the biases; run a short causal
//     convolution over time on every channel (y_t = sum_j w[c, j] u_(t - taps + 1 + j), zeros in front of the sequence; the
//     sequence's last taps - 1 inputs live in its state row between steps); normalise the WHOLE q and the whole k of the
//     token (x / sqrt(mean(x^2) + eps) * w over all heads at once); rotate the first rot_dims numbers of every head, members
//     (2i, 2i + 1) of a pair, by the token's position; write q for the attention kernel and append k and v to the paged
//     cache.  Every stage is optional (a null pointer or a zero size turns it off).  Sums, statistics and angles are 32-bit.
//   * fg_conv_state_update: after it, the sequences' new last taps - 1 inputs go to their state rows.
//   * fg_latent_append: a token's latent (normalised) goes to the value pool, its shared rotated key part to the key pool.
//   * fg_rope_pairs: rotation of adjacent pairs on a slice of every head, from one buffer into another.
//   * fg_rmsnorm_strided: RMS norm of float32 rows that are a slice of a wider matrix.
//   * fg_head_gemm: one small contraction per head, C[m, h, :] = A[m, h, :] W_h^T (or W_h), optionally times sigmoid(gate).
#include "common.cuh"

#define PREP_THREADS 256

// four neighbours of a row: 16 bytes of float32, or 8 of bfloat16
template <typename T> __device__ __forceinline__ void put4(T *dst, const float *p);
template <> __device__ __forceinline__ void put4<float>(float *dst, const float *p) { *(float4 *)dst = *(const float4 *)p; }
template <> __device__ __forceinline__ void put4<bf16>(bf16 *dst, const float *p) {
    const float4 v = *(const float4 *)p;
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *(uint2 *)dst = make_uint2(*(uint32_t *)&lo, *(uint32_t *)&hi);
}

// cos/sin: [positions, tbl_half] float32, column i = pair i.
// VEC: no convolution, and rows, heads and pools allow accesses of four numbers.
template <typename T, bool VEC>
__global__ void __launch_bounds__(1024)
qkv_prepare_kernel(const float *__restrict__ proj, int ld, const float *__restrict__ bias, const float *__restrict__ conv_w, int taps,
                   const float *__restrict__ conv_state, const float *__restrict__ qn_w, const float *__restrict__ kn_w, float eps,
                   const float *__restrict__ cos_t, const float *__restrict__ sin_t, int tbl_half, int rot_dims,
                   const int *__restrict__ positions, const int *__restrict__ row_seq, const int *__restrict__ cu_rows,
                   const int *__restrict__ slots, const int *__restrict__ block_table, int table_width, T *__restrict__ q_out, int ldq,
                   T *__restrict__ k_pool, T *__restrict__ v_pool, int H, int KV, int VH, int hd, int hdv, int page_size, int norm_per_head,
                   int rot_halves, int v_from_k) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[32];
    pdl_launch_dependents_small_step(gridDim.x);
    pdl_wait();
    const int m = blockIdx.x, tid = threadIdx.x, nthr = blockDim.x;
    const int Cq = H * hd, Ck = KV * hd, C = Cq + Ck + (v_from_k ? 0 : VH * hdv);
    const int seq = row_seq[m], pos = positions[m];
    const int i_step = m - cu_rows[seq];                 // the token's index among the step's tokens of its sequence
    const float *mine = proj + (size_t)m * ld;
    if (VEC) {
        for (int c = tid * 4; c < C; c += nthr * 4) {
            float4 v = *(const float4 *)(mine + c);
            if (bias) { const float4 b = *(const float4 *)(bias + c); v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
            *(float4 *)(row + c) = v;
        }
    } else if (conv_w) {
        const float *st = conv_state + (size_t)slots[seq] * (taps - 1) * C;
        for (int c = tid; c < C; c += nthr) {
            const float b = bias ? bias[c] : 0.f;
            float acc = 0.f;
            for (int j = 0; j < taps; j++) {
                const int back = taps - 1 - j;           // the input `back` tokens ago
                float u;
                if (back <= i_step) u = proj[(size_t)(m - back) * ld + c] + b;
                else u = st[(size_t)(taps - 1 - (back - i_step)) * C + c];      // from before this step (zeros before the sequence)
                acc = fmaf(conv_w[(size_t)c * taps + j], u, acc);
            }
            row[c] = acc;
        }
    } else {
        for (int c = tid; c < C; c += nthr) row[c] = mine[c] + (bias ? bias[c] : 0.f);
    }
    __syncthreads();
    if (v_from_k && v_pool) {
        // the values are the keys as projected (bias included), before norm and rotation
        const int page = block_table[(size_t)seq * table_width + pos / page_size], off = pos % page_size;
        if (VEC) {
            for (int c = tid * 4; c < Ck; c += nthr * 4) {
                const int vh = c / hdv, d = c - vh * hdv;
                put4<T>(v_pool + (((size_t)page * VH + vh) * page_size + off) * hdv + d, row + Cq + c);
            }
        } else {
            for (int c = tid; c < Ck; c += nthr) {
                const int vh = c / hdv, d = c - vh * hdv;
                v_pool[(((size_t)page * VH + vh) * page_size + off) * hdv + d] = from_f32<T>(row[Cq + c]);
            }
        }
        __syncthreads();
    }
    if (qn_w && norm_per_head) {
        // every head of q and of k by itself: x / sqrt(mean(x^2) + eps) * w with ONE weight vector [hd] for all heads of q and
        // one for all heads of k; a warp takes a head, its lanes the head's numbers, the sum by a shuffle tree
        const int warp = tid >> 5, lane = tid & 31, n_warps = nthr >> 5;
        for (int head = warp; head < H + KV; head += n_warps) {
            float *p = row + (size_t)head * hd;
            const float *w = head < H ? qn_w : kn_w;
            float ss = 0.f;
            for (int d = lane; d < hd; d += 32) ss = fmaf(p[d], p[d], ss);
            ss = warp_sum(ss);
            const float inv = 1.0f / sqrtf(ss / (float)hd + eps);
            for (int d = lane; d < hd; d += 32) p[d] = p[d] * inv * w[d];
        }
        __syncthreads();
    } else if (qn_w) {
        float sq = 0.f, sk = 0.f;
        for (int c = tid; c < Cq; c += nthr) sq = fmaf(row[c], row[c], sq);
        for (int c = tid; c < Ck; c += nthr) sk = fmaf(row[Cq + c], row[Cq + c], sk);
        sq = block_sum(sq, scratch);
        sk = block_sum(sk, scratch);
        const float iq = 1.0f / sqrtf(sq / (float)Cq + eps), ik = 1.0f / sqrtf(sk / (float)Ck + eps);
        for (int c = tid; c < Cq; c += nthr) row[c] = row[c] * iq * qn_w[c];
        for (int c = tid; c < Ck; c += nthr) row[Cq + c] = row[Cq + c] * ik * kn_w[c];
        __syncthreads();
    }
    const int rh = rot_dims / 2;
    if (rh > 0) {
        const float *cs = cos_t + (size_t)pos * tbl_half, *sn = sin_t + (size_t)pos * tbl_half;
        for (int e = tid; e < (H + KV) * rh; e += nthr) {
            const int head = e / rh, i = e - head * rh;
            // q heads and k heads lie one after another, all of size hd; a pair is (2i, 2i + 1), or (i, i + rot_dims / 2)
            float *p = row + (size_t)head * hd + (rot_halves ? i : 2 * i);
            const int other = rot_halves ? rh : 1;
            const float a = p[0], b = p[other], c = cs[i], s = sn[i];
            p[0] = a * c - b * s;
            p[other] = b * c + a * s;
        }
        __syncthreads();
    }
    if (VEC) {
        for (int c = tid * 4; c < Cq; c += nthr * 4) put4<T>(q_out + (size_t)m * ldq + c, row + c);
        if (!k_pool) return;
        const int page = block_table[(size_t)seq * table_width + pos / page_size], off = pos % page_size;
        for (int c = tid * 4; c < Ck; c += nthr * 4) {
            const int kvh = c / hd, d = c - kvh * hd;
            put4<T>(k_pool + (((size_t)page * KV + kvh) * page_size + off) * hd + d, row + Cq + c);
        }
        for (int c = tid * 4; c < (v_from_k ? 0 : VH * hdv); c += nthr * 4) {
            const int vh = c / hdv, d = c - vh * hdv;
            put4<T>(v_pool + (((size_t)page * VH + vh) * page_size + off) * hdv + d, row + Cq + Ck + c);
        }
        return;
    }
    for (int c = tid; c < Cq; c += nthr) q_out[(size_t)m * ldq + c] = from_f32<T>(row[c]);
    if (k_pool) {
        const int page = block_table[(size_t)seq * table_width + pos / page_size], off = pos % page_size;
        for (int c = tid; c < Ck; c += nthr) {
            const int kvh = c / hd, d = c - kvh * hd;
            k_pool[(((size_t)page * KV + kvh) * page_size + off) * hd + d] = from_f32<T>(row[Cq + c]);
        }
        for (int c = tid; c < (v_from_k ? 0 : VH * hdv); c += nthr) {
            const int vh = c / hdv, d = c - vh * hdv;
            v_pool[(((size_t)page * VH + vh) * page_size + off) * hdv + d] = from_f32<T>(row[Cq + Ck + c]);
        }
    }
}

// state[slot][j][c], j < taps - 1: the sequence's input (projection + bias) of taps - 1 - j tokens before its end
__global__ void conv_state_update_kernel(const float *__restrict__ proj, int ld, const float *__restrict__ bias, int taps,
                                         float *__restrict__ conv_state, const int *__restrict__ cu_rows, const int *__restrict__ slots,
                                         int C) {
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int r0 = cu_rows[seq], n = cu_rows[seq + 1] - r0;
    if (n <= 0) return;
    float *st = conv_state + (size_t)slots[seq] * (taps - 1) * C;
    const float b = bias ? bias[c] : 0.f;
    for (int j = 0; j < taps - 1; j++) {
        const int idx = n - (taps - 1) + j;              // index among the step's tokens
        // an older input moves up: it is read at j + n > j, before anything at or above it is written
        st[(size_t)j * C + c] = idx >= 0 ? proj[(size_t)(r0 + idx) * ld + c] + b : st[(size_t)(j + n) * C + c];
    }
}

template <typename T>
__global__ void __launch_bounds__(PREP_THREADS)
latent_append_kernel(const float *__restrict__ kv, int ld, const float *__restrict__ norm_w, float eps, const float *__restrict__ cos_t,
                     const float *__restrict__ sin_t, int tbl_half, const int *__restrict__ positions, const int *__restrict__ row_seq,
                     const int *__restrict__ block_table, int table_width, T *__restrict__ k_pool, T *__restrict__ v_pool, int rank,
                     int rot_dim, int page_size) {
    __shared__ float scratch[32];
    pdl_launch_dependents_small_step(gridDim.x);
    pdl_wait();
    const int m = blockIdx.x, tid = threadIdx.x;
    const int pos = positions[m];
    const int page = block_table[(size_t)row_seq[m] * table_width + pos / page_size], off = pos % page_size;
    const float *src = kv + (size_t)m * ld;
    float ss = 0.f;
    for (int c = tid; c < rank; c += PREP_THREADS) ss = fmaf(src[c], src[c], ss);
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)rank + eps);
    T *lat = v_pool + ((size_t)page * page_size + off) * rank;
    for (int c = tid; c < rank; c += PREP_THREADS) lat[c] = from_f32<T>(src[c] * inv * norm_w[c]);
    T *kr = k_pool + ((size_t)page * page_size + off) * rot_dim;
    const float *cs = cos_t + (size_t)pos * tbl_half, *sn = sin_t + (size_t)pos * tbl_half;
    for (int i = tid; i < rot_dim / 2; i += PREP_THREADS) {
        const float a = src[rank + 2 * i], b = src[rank + 2 * i + 1], c = cs[i], s = sn[i];
        kr[2 * i] = from_f32<T>(a * c - b * s);
        kr[2 * i + 1] = from_f32<T>(b * c + a * s);
    }
}

// out[m, h * out_stride + out_off + (0 .. dims)) = rotation of in[m, h * in_stride + in_off + (0 .. dims))
template <typename T>
__global__ void rope_pairs_kernel(const float *__restrict__ in, int ld_in, int in_stride, int in_off, T *__restrict__ out, int ld_out,
                                  int out_stride, int out_off, const int *__restrict__ positions, const float *__restrict__ cos_t,
                                  const float *__restrict__ sin_t, int tbl_half, int H, int dims) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, rh = dims / 2;
    const int pos = positions[m];
    const float *cs = cos_t + (size_t)pos * tbl_half, *sn = sin_t + (size_t)pos * tbl_half;
    for (int e = threadIdx.x; e < H * rh; e += blockDim.x) {
        const int h = e / rh, i = e - h * rh;
        const float *p = in + (size_t)m * ld_in + (size_t)h * in_stride + in_off + 2 * i;
        T *o = out + (size_t)m * ld_out + (size_t)h * out_stride + out_off + 2 * i;
        const float a = p[0], b = p[1], c = cs[i], s = sn[i];
        o[0] = from_f32<T>(a * c - b * s);
        o[1] = from_f32<T>(b * c + a * s);
    }
}

template <typename T>
__global__ void __launch_bounds__(PREP_THREADS)
rmsnorm_strided_kernel(const float *__restrict__ x, int ldx, const float *__restrict__ w, T *__restrict__ out, int ldo, int E, float eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents_small_step(gridDim.x);
    pdl_wait();
    const float *src = x + (size_t)blockIdx.x * ldx;
    float ss = 0.f;
    for (int c = threadIdx.x; c < E; c += PREP_THREADS) ss = fmaf(src[c], src[c], ss);
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)E + eps);
    for (int c = threadIdx.x; c < E; c += PREP_THREADS) out[(size_t)blockIdx.x * ldo + c] = from_f32<T>(src[c] * inv * w[c]);
}

// C[m, h * c_stride + n] = sum_k A[m, h * a_stride + k] * W_h[n, k]; W_h[n, k] is w[(h * N + n) * ldw + k], or, transposed,
// w[(h * K + k) * ldw + n].  gate (float32, [M, ldg], column h * N + n): the result is multiplied by sigmoid(gate).
// 64 x 64 output tiles, 16 x 16 threads of 4 x 4 outputs, K in steps of 16; sums run along k in order.
#define HG_T 64
#define HG_K 16
__global__ void __launch_bounds__(256)
head_gemm_kernel(const void *__restrict__ A, int a_dtype, int lda, int a_stride, const void *__restrict__ W, int w_dtype, int ldw,
                 int transposed, void *__restrict__ Cm, int c_dtype, int ldc, int c_stride, const float *__restrict__ gate, int ldg, int M,
                 int N, int K) {
    __shared__ float As[HG_K][HG_T + 1], Ws[HG_K][HG_T + 1];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.z, m0 = blockIdx.y * HG_T, n0 = blockIdx.x * HG_T;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += HG_K) {
        for (int e = threadIdx.x; e < HG_T * HG_K; e += 256) {
            const int r = e / HG_K, k = e - r * HG_K;      // k fastest: rows of A and of W are read along k
            const int m = m0 + r, n = n0 + r;
            As[k][r] = (m < M && k0 + k < K) ? load_as(A, a_dtype, (size_t)m * lda + (size_t)h * a_stride + k0 + k) : 0.f;
            if (!transposed) Ws[k][r] = (n < N && k0 + k < K) ? load_as(W, w_dtype, ((size_t)h * N + n) * ldw + k0 + k) : 0.f;
        }
        if (transposed)
            for (int e = threadIdx.x; e < HG_T * HG_K; e += 256) {
                const int k = e / HG_T, r = e - k * HG_T;  // n fastest: a row of the stored matrix runs along n
                const int n = n0 + r;
                Ws[k][r] = (n < N && k0 + k < K) ? load_as(W, w_dtype, ((size_t)h * K + k0 + k) * ldw + n) : 0.f;
            }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < HG_K; k++) {
            float a[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { a[i] = As[k][ty * 4 + i]; w[i] = Ws[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (m >= M || n >= N) continue;
            float v = acc[i][j];
            if (gate) v *= 1.0f / (1.0f + expf(-gate[(size_t)m * ldg + (size_t)h * N + n]));
            store_as(Cm, c_dtype, (size_t)m * ldc + (size_t)h * c_stride + n, v);
        }
}

// The same contraction for a few rows (a decode step): every weight is read once, in 16-byte or paired accesses, for all rows.
// TRANSPOSED (a stored row runs along n): a thread owns two neighbouring outputs and, for bfloat16 weights, a quarter of the sum
// over k, the four quarters being added in order in shared memory; for float32 weights the whole sum in order, as the tiled
// kernel adds it.  Else (a stored row runs along k): a warp owns two outputs, its lanes lie along
// k, and the sums meet in a shuffle tree.  RM: rows the registers hold (M <= RM).  vec: the sizes allow the wide accesses.
#define HV_ROWS 16
#define HV_COLS 128                                     // outputs of 64 threads, transposed
template <typename TW> struct HvPair;
template <> struct HvPair<float> { static __device__ __forceinline__ float2 load(const float *p) { return *(const float2 *)p; } };
template <> struct HvPair<bf16> { static __device__ __forceinline__ float2 load(const bf16 *p) { return __bfloat1622float2(*(const __nv_bfloat162 *)p); } };

template <typename TW, bool TRANSPOSED, int RM>
__global__ void __launch_bounds__(256)
head_gemv_kernel(const void *__restrict__ A, int a_dtype, int lda, int a_stride, const TW *__restrict__ W, int ldw,
                 void *__restrict__ Cm, int c_dtype, int ldc, int c_stride, const float *__restrict__ gate, int ldg, int M, int N, int K,
                 int vec) {
    extern __shared__ __align__(16) float as[];         // transposed: [K][RM], then the quarters' sums; else [RM][KP]
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, tid = threadIdx.x, KP = (K + 3) / 4 * 4;
    for (int e = tid; e < RM * K; e += 256) {
        const int m = e / K, k = e - m * K;
        as[TRANSPOSED ? k * RM + m : m * KP + k] = m < M ? load_as(A, a_dtype, (size_t)m * lda + (size_t)h * a_stride + k) : 0.f;
    }
    __syncthreads();
    float acc[2][RM];
#pragma unroll
    for (int m = 0; m < RM; m++) acc[0][m] = acc[1][m] = 0.f;
    auto store = [&](int m, int n, float v) {
        if (gate) v *= 1.0f / (1.0f + expf(-gate[(size_t)m * ldg + (size_t)h * N + n]));
        store_as(Cm, c_dtype, (size_t)m * ldc + (size_t)h * c_stride + n, v);
    };
    if (TRANSPOSED) {
        constexpr bool QUARTERS = sizeof(TW) == 2;
        const int grp = tid >> 6, n = (QUARTERS ? blockIdx.x : blockIdx.x * 4 + grp) * HV_COLS + 2 * (tid & 63), KQ = QUARTERS ? (K + 3) / 4 : K,
                  k_begin = QUARTERS ? grp * KQ : 0, k_end = min(K, k_begin + KQ);
        const TW *w0 = W + (size_t)h * K * ldw + n;
        if (n < N) {
            for (int k0 = k_begin; k0 < k_end; k0 += 8) {
                float2 w[8];                                // eight weights' rows on their way before the first is used
#pragma unroll
                for (int u = 0; u < 8; u++) {
                    const TW *p = w0 + (size_t)min(k0 + u, K - 1) * ldw;
                    if (vec) w[u] = HvPair<TW>::load(p);
                    else w[u] = make_float2(to_f32<TW>(p[0]), n + 1 < N ? to_f32<TW>(p[1]) : 0.f);
                }
#pragma unroll
                for (int u = 0; u < 8; u++) {
                    if (k0 + u >= k_end) break;
                    const float4 *x4 = (const float4 *)(as + (size_t)(k0 + u) * RM);
#pragma unroll
                    for (int q = 0; q < RM / 4; q++) {
                        const float4 x = x4[q];
                        acc[0][4 * q] = fmaf(x.x, w[u].x, acc[0][4 * q]); acc[1][4 * q] = fmaf(x.x, w[u].y, acc[1][4 * q]);
                        acc[0][4 * q + 1] = fmaf(x.y, w[u].x, acc[0][4 * q + 1]); acc[1][4 * q + 1] = fmaf(x.y, w[u].y, acc[1][4 * q + 1]);
                        acc[0][4 * q + 2] = fmaf(x.z, w[u].x, acc[0][4 * q + 2]); acc[1][4 * q + 2] = fmaf(x.z, w[u].y, acc[1][4 * q + 2]);
                        acc[0][4 * q + 3] = fmaf(x.w, w[u].x, acc[0][4 * q + 3]); acc[1][4 * q + 3] = fmaf(x.w, w[u].y, acc[1][4 * q + 3]);
                    }
                }
            }
        }
        if (!QUARTERS) {
#pragma unroll
            for (int m = 0; m < RM; m++) {
                if (m >= M || n >= N) break;
                store(m, n, acc[0][m]);
                if (n + 1 < N) store(m, n + 1, acc[1][m]);
            }
            return;
        }
        __syncthreads();                                    // the rows are read; their memory takes the sums [4][RM][HV_COLS]
#pragma unroll
        for (int m = 0; m < RM; m++) *(float2 *)(as + ((size_t)grp * RM + m) * HV_COLS + 2 * (tid & 63)) = make_float2(acc[0][m], acc[1][m]);
        __syncthreads();
        for (int e = tid; e < M * HV_COLS; e += 256) {
            const int m = e / HV_COLS, c = e - m * HV_COLS, nn = blockIdx.x * HV_COLS + c;
            if (nn >= N) continue;
            float v = 0.f;
#pragma unroll
            for (int g = 0; g < 4; g++) v += as[((size_t)g * RM + m) * HV_COLS + c];
            store(m, nn, v);
        }
    } else {
        const int lane = tid & 31, n = (blockIdx.x * 8 + (tid >> 5)) * 2;
        if (n >= N) return;
        constexpr int VEC = 16 / (int)sizeof(TW);
        const TW *w0 = W + ((size_t)h * N + n) * ldw, *w1 = n + 1 < N ? w0 + ldw : w0;
        if (vec) {
#pragma unroll 2
            for (int k = lane * VEC; k < K; k += 32 * VEC) {
                const uint4 r0 = *(const uint4 *)(w0 + k), r1 = *(const uint4 *)(w1 + k);
                const TW *e0 = (const TW *)&r0, *e1 = (const TW *)&r1;
#pragma unroll
                for (int m = 0; m < RM; m++) {
                    float x[VEC];
#pragma unroll
                    for (int i = 0; i < VEC; i += 4) *(float4 *)(x + i) = *(const float4 *)(as + m * KP + k + i);
#pragma unroll
                    for (int i = 0; i < VEC; i++) {
                        acc[0][m] = fmaf(x[i], to_f32<TW>(e0[i]), acc[0][m]);
                        acc[1][m] = fmaf(x[i], to_f32<TW>(e1[i]), acc[1][m]);
                    }
                }
            }
        } else {
            for (int k = lane; k < K; k += 32) {
                const float a = to_f32<TW>(w0[k]), b = to_f32<TW>(w1[k]);
#pragma unroll
                for (int m = 0; m < RM; m++) { acc[0][m] = fmaf(as[m * KP + k], a, acc[0][m]); acc[1][m] = fmaf(as[m * KP + k], b, acc[1][m]); }
            }
        }
        // sums of 2 RM numbers: at every exchange a lane keeps half of them, and ends with one (RM = 16) or one twice over (RM = 8)
        float v[2 * RM];
#pragma unroll
        for (int m = 0; m < RM; m++) { v[m] = acc[0][m]; v[RM + m] = acc[1][m]; }
#pragma unroll
        for (int o = RM; o > 0; o >>= 1) {
            const bool up = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < o; i++) {
                const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
        if (RM == 8) v[0] += __shfl_xor_sync(0xffffffffu, v[0], 16);
        const int m = lane & (RM - 1), c = (lane / RM) & 1;
        if (lane < 2 * RM && m < M && n + c < N) store(m, n + c, v[0]);
    }
}

// norm_per_head: the norm weights are [hd] and every head of q and of k is normalised by itself (else: [H * hd] / [KV * hd], the
// whole of q and of k at once); rot_halves: a rotated pair is (i, i + rot_dims / 2) of a head (else (2i, 2i + 1)); v_heads (0: KV):
// heads of values, where several key heads share one; v_from_k: there is no value projection, the values are the keys as projected
extern "C" int fg_qkv_prepare_ext(const float *proj, int ld, const float *bias, const float *conv_w, int taps, const float *conv_state,
                                  const float *qn_w, const float *kn_w, float eps, const float *cos_t, const float *sin_t, int tbl_half,
                                  int rot_dims, const int *positions, const int *row_seq, const int *cu_rows, const int *slots,
                                  const int *block_table, int table_width, void *q_out, int ldq, void *k_pool, void *v_pool, int dtype, int M,
                                  int H, int KV, int hd, int hdv, int page_size, int norm_per_head, int rot_halves, int v_heads, int v_from_k,
                                  cudaStream_t stream) {
    if (M <= 0) return 0;
    const int VH = v_heads > 0 ? v_heads : KV;
    if (v_from_k && (conv_w || VH != KV || hdv != hd)) return FG_ERR_BAD_SIZE;
    if (H <= 0 || KV <= 0 || hd <= 0 || hdv <= 0 || rot_dims < 0 || rot_dims % 2 || rot_dims > hd || rot_dims / 2 > tbl_half) return FG_ERR_BAD_SIZE;
    if (conv_w && (taps < 1 || (taps > 1 && !conv_state))) return FG_ERR_BAD_SIZE;
    if ((qn_w == nullptr) != (kn_w == nullptr)) return FG_ERR_BAD_SIZE;
    const int C_all = H * hd + KV * hd + (v_from_k ? 0 : VH * hdv);
    const size_t smem = (size_t)C_all * sizeof(float);
    if (smem > 200 * 1024) return FG_ERR_BAD_SIZE;
    // few rows (a decode step) leave most of the GPU idle: a row's channels are then spread over more threads
    const int threads = (M < 64 && C_all >= 2048) ? 1024 : PREP_THREADS;
    const bool vec = !conv_w && hd % 4 == 0 && hdv % 4 == 0 && ld % 4 == 0 && ldq % 4 == 0 &&
                     ((((uintptr_t)proj) | ((uintptr_t)bias) | ((uintptr_t)q_out) | ((uintptr_t)k_pool) | ((uintptr_t)v_pool)) & 15) == 0;
#define PREP_RUN(T, VEC) do { \
        static FgPerDevice setup; \
        if (smem > 48 * 1024 && fg_needs_setup(setup)) { \
            cudaError_t e = cudaFuncSetAttribute(qkv_prepare_kernel<T, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
            if (e != cudaSuccess) return (int)e; \
        } \
        return fg_launch(qkv_prepare_kernel<T, VEC>, dim3(M), dim3(threads), smem, stream, proj, ld, bias, conv_w, taps, conv_state, qn_w, kn_w, \
                         eps, cos_t, sin_t, tbl_half, rot_dims, positions, row_seq, cu_rows, slots, block_table, table_width, (T *)q_out, \
                         ldq, (T *)k_pool, (T *)v_pool, H, KV, VH, hd, hdv, page_size, norm_per_head, rot_halves, v_from_k); } while (0)
    if (dtype == FG_F32) {
        if (vec) PREP_RUN(float, true);
        PREP_RUN(float, false);
    }
    if (dtype == FG_BF16) {
        if (vec) PREP_RUN(bf16, true);
        PREP_RUN(bf16, false);
    }
#undef PREP_RUN
    return FG_ERR_BAD_DTYPE;
}

extern "C" int fg_qkv_prepare(const float *proj, int ld, const float *bias, const float *conv_w, int taps, const float *conv_state,
                              const float *qn_w, const float *kn_w, float eps, const float *cos_t, const float *sin_t, int tbl_half,
                              int rot_dims, const int *positions, const int *row_seq, const int *cu_rows, const int *slots,
                              const int *block_table, int table_width, void *q_out, int ldq, void *k_pool, void *v_pool, int dtype, int M,
                              int H, int KV, int hd, int hdv, int page_size, cudaStream_t stream) {
    return fg_qkv_prepare_ext(proj, ld, bias, conv_w, taps, conv_state, qn_w, kn_w, eps, cos_t, sin_t, tbl_half, rot_dims, positions, row_seq,
                              cu_rows, slots, block_table, table_width, q_out, ldq, k_pool, v_pool, dtype, M, H, KV, hd, hdv, page_size, 0, 0, 0, 0, stream);
}

// ------------------------------------------------------------------ the difference of two maps' outputs
// maps [M, 2 H * dv] float32, heads in the order [key head g][map][head i of the group]: with a1, a2 the two maps' outputs of a head,
// o = a1 - lambda a2, out = o / sqrt(mean(o^2) + eps) * gain over the head's dv values; out's heads are g * R + i.  A warp a head.
template <typename T, bool VEC>
__global__ void __launch_bounds__(PREP_THREADS)
differential_combine_kernel(const float *__restrict__ maps, int ld, T *__restrict__ out, int ldo, int H, int R, int dv, float lambda, float eps,
                            float gain) {
    pdl_launch_dependents_small_step(gridDim.x);
    pdl_wait();
    const int m = blockIdx.x, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    for (int h = blockIdx.y * n_warps + (threadIdx.x >> 5); h < H; h += gridDim.y * n_warps) {
        const int g = h / R, i = h - g * R;
        const float *a1 = maps + (size_t)m * ld + (size_t)(2 * g * R + i) * dv, *a2 = a1 + (size_t)R * dv;
        T *o = out + (size_t)m * ldo + (size_t)h * dv;
        float ss = 0.f;
        if (VEC) {
            for (int d = lane * 4; d < dv; d += 128) {
                const float4 x = *(const float4 *)(a1 + d), y = *(const float4 *)(a2 + d);
                const float p = fmaf(-lambda, y.x, x.x), q = fmaf(-lambda, y.y, x.y), r = fmaf(-lambda, y.z, x.z), s = fmaf(-lambda, y.w, x.w);
                ss += p * p; ss += q * q; ss += r * r; ss += s * s;
            }
        } else {
            for (int d = lane; d < dv; d += 32) { const float p = fmaf(-lambda, a2[d], a1[d]); ss += p * p; }
        }
        const float inv = gain / sqrtf(warp_sum(ss) / (float)dv + eps);
        if (VEC) {
            for (int d = lane * 4; d < dv; d += 128) {
                const float4 x = *(const float4 *)(a1 + d), y = *(const float4 *)(a2 + d);
                const float p = fmaf(-lambda, y.x, x.x) * inv, q = fmaf(-lambda, y.y, x.y) * inv, r = fmaf(-lambda, y.z, x.z) * inv, s = fmaf(-lambda, y.w, x.w) * inv;
                if (sizeof(T) == 4) *(float4 *)(o + d) = make_float4(p, q, r, s);
                else {
                    __nv_bfloat162 lo = __floats2bfloat162_rn(p, q), hi = __floats2bfloat162_rn(r, s);
                    *(uint2 *)(o + d) = make_uint2(*(uint32_t *)&lo, *(uint32_t *)&hi);
                }
            }
        } else {
            for (int d = lane; d < dv; d += 32) o[d] = from_f32<T>(fmaf(-lambda, a2[d], a1[d]) * inv);
        }
    }
}

extern "C" int fg_differential_combine(const float *maps, int ld, void *out, int out_dtype, int ldo, int M, int H, int KV, int dv, float lambda,
                                       float eps, float gain, cudaStream_t stream) {
    if (M <= 0) return 0;
    if (H <= 0 || KV <= 0 || H % KV || dv <= 0) return FG_ERR_BAD_SIZE;
    const bool vec = dv % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && ((((uintptr_t)maps) | ((uintptr_t)out)) & 15) == 0;
    const dim3 grid(M, (H + 7) / 8);
#define DIFF_LAUNCH(T, VEC) fg_launch(differential_combine_kernel<T, VEC>, grid, dim3(PREP_THREADS), 0, stream, maps, ld, (T *)out, ldo, H, H / KV, dv, lambda, \
                                      eps, gain)
    if (out_dtype == FG_F32) return vec ? DIFF_LAUNCH(float, true) : DIFF_LAUNCH(float, false);
    if (out_dtype == FG_BF16) return vec ? DIFF_LAUNCH(bf16, true) : DIFF_LAUNCH(bf16, false);
#undef DIFF_LAUNCH
    return FG_ERR_BAD_DTYPE;
}

// ------------------------------------------------------------------ a gate per head on the heads' outputs
// x[m, h * DV + j] *= sigmoid(gate[m, h]) in place (gate float32, one number a head and row; null: no gate), and `pad` columns
// behind the heads are set to (1, 0, 0, ...): with the output projection's bias stored as column H * DV of its matrix, the
// projection adds the bias in the same pass.
template <typename T>
__global__ void head_gate_kernel(T *__restrict__ x, int ldx, const float *__restrict__ gate, int ldg, int H, int DV, int pad, int vec) {
    extern __shared__ float head_gate_sig[];        // the row's H gates
    // (no early release of the successor: this kernel stands between two tensor-memory contractions, and the second must not
    // start beside the first while this one sits resident and waiting; the successor starts when this kernel has finished)
    pdl_wait();
    const int m = blockIdx.x;
    T *row = x + (size_t)m * ldx;
    if (gate) {
        for (int h = threadIdx.x; h < H; h += blockDim.x) head_gate_sig[h] = 1.0f / (1.0f + expf(-gate[(size_t)m * ldg + h]));
        __syncthreads();
        if (vec) {
            // 16 bytes a thread; DV is a multiple of the run, so a run lies in one head
            constexpr int PER = 16 / sizeof(T);
            for (int e = threadIdx.x * PER; e < H * DV; e += blockDim.x * PER) {
                const float g = head_gate_sig[e / DV];
                uint4 raw = *reinterpret_cast<const uint4 *>(row + e);
                T *v = reinterpret_cast<T *>(&raw);
#pragma unroll
                for (int i = 0; i < PER; i++) v[i] = from_f32<T>(to_f32<T>(v[i]) * g);
                *reinterpret_cast<uint4 *>(row + e) = raw;
            }
        } else {
            for (int e = threadIdx.x; e < H * DV; e += blockDim.x) row[e] = from_f32<T>(to_f32<T>(row[e]) * head_gate_sig[e / DV]);
        }
    }
    for (int e = threadIdx.x; e < pad; e += blockDim.x) row[H * DV + e] = from_f32<T>(e == 0 ? 1.0f : 0.0f);
}

extern "C" int fg_head_gate(void *x, int ldx, int dtype, const float *gate, int ldg, int M, int H, int DV, int pad, cudaStream_t stream) {
    if (M <= 0 || (!gate && pad <= 0)) return 0;
    if (H * DV + pad > ldx || H > 8192) return FG_ERR_BAD_SIZE;
    const int threads = H * DV >= 4096 ? 256 : 128;
    const size_t smem = (size_t)H * sizeof(float);
    const int per = dtype == FG_F32 ? 4 : 8;
    const int vec = (DV % per == 0 && ldx % per == 0 && ((uintptr_t)x & 15) == 0) ? 1 : 0;
    if (dtype == FG_F32) return fg_launch(head_gate_kernel<float>, dim3(M), dim3(threads), smem, stream, (float *)x, ldx, gate, ldg, H, DV, pad, vec);
    if (dtype == FG_BF16) return fg_launch(head_gate_kernel<bf16>, dim3(M), dim3(threads), smem, stream, (bf16 *)x, ldx, gate, ldg, H, DV, pad, vec);
    return FG_ERR_BAD_DTYPE;
}

extern "C" int fg_conv_state_update(const float *proj, int ld, const float *bias, int taps, float *conv_state, const int *cu_rows,
                                    const int *slots, int n_seq, int C, cudaStream_t stream) {
    if (n_seq <= 0 || taps <= 1) return 0;
    if (C <= 0) return FG_ERR_BAD_SIZE;
    return fg_launch(conv_state_update_kernel, dim3(n_seq, (C + 255) / 256), dim3(256), 0, stream, proj, ld, bias, taps, conv_state, cu_rows, slots, C);
}

extern "C" int fg_latent_append(const float *kv, int ld, const float *norm_w, float eps, const float *cos_t, const float *sin_t, int tbl_half,
                                const int *positions, const int *row_seq, const int *block_table, int table_width, void *k_pool,
                                void *v_pool, int dtype, int M, int rank, int rot_dim, int page_size, cudaStream_t stream) {
    if (M <= 0) return 0;
    if (rank <= 0 || rot_dim <= 0 || rot_dim % 2 || rot_dim / 2 > tbl_half) return FG_ERR_BAD_SIZE;
    if (dtype == FG_F32)
        return fg_launch(latent_append_kernel<float>, dim3(M), dim3(PREP_THREADS), 0, stream, kv, ld, norm_w, eps, cos_t, sin_t, tbl_half, positions,
                         row_seq, block_table, table_width, (float *)k_pool, (float *)v_pool, rank, rot_dim, page_size);
    if (dtype == FG_BF16)
        return fg_launch(latent_append_kernel<bf16>, dim3(M), dim3(PREP_THREADS), 0, stream, kv, ld, norm_w, eps, cos_t, sin_t, tbl_half, positions,
                         row_seq, block_table, table_width, (bf16 *)k_pool, (bf16 *)v_pool, rank, rot_dim, page_size);
    return FG_ERR_BAD_DTYPE;
}

extern "C" int fg_rope_pairs(const float *in, int ld_in, int in_stride, int in_off, void *out, int out_dtype, int ld_out, int out_stride,
                             int out_off, const int *positions, const float *cos_t, const float *sin_t, int tbl_half, int M, int H, int dims,
                             cudaStream_t stream) {
    if (M <= 0 || dims <= 0) return 0;
    if (dims % 2 || dims / 2 > tbl_half || H <= 0) return FG_ERR_BAD_SIZE;
    const int threads = H * dims / 2 >= 256 ? 256 : 64;
    if (out_dtype == FG_F32)
        return fg_launch(rope_pairs_kernel<float>, dim3(M), dim3(threads), 0, stream, in, ld_in, in_stride, in_off, (float *)out, ld_out, out_stride,
                         out_off, positions, cos_t, sin_t, tbl_half, H, dims);
    if (out_dtype == FG_BF16)
        return fg_launch(rope_pairs_kernel<bf16>, dim3(M), dim3(threads), 0, stream, in, ld_in, in_stride, in_off, (bf16 *)out, ld_out, out_stride,
                         out_off, positions, cos_t, sin_t, tbl_half, H, dims);
    return FG_ERR_BAD_DTYPE;
}

extern "C" int fg_rmsnorm_strided(const float *x, int ldx, const float *w, void *out, int out_dtype, int ldo, int R, int E, float eps,
                                  cudaStream_t stream) {
    if (R <= 0) return 0;
    if (E <= 0) return FG_ERR_BAD_SIZE;
    if (out_dtype == FG_F32) return fg_launch(rmsnorm_strided_kernel<float>, dim3(R), dim3(PREP_THREADS), 0, stream, x, ldx, w, (float *)out, ldo, E, eps);
    if (out_dtype == FG_BF16) return fg_launch(rmsnorm_strided_kernel<bf16>, dim3(R), dim3(PREP_THREADS), 0, stream, x, ldx, w, (bf16 *)out, ldo, E, eps);
    return FG_ERR_BAD_DTYPE;
}

extern "C" int fg_head_gemm(const void *A, int a_dtype, int lda, int a_stride, const void *W, int w_dtype, int ldw, int transposed, void *C,
                            int c_dtype, int ldc, int c_stride, const float *gate, int ldg, int M, int N, int K, int H, cudaStream_t stream) {
    if (M <= 0 || N <= 0 || H <= 0) return 0;
    if (K <= 0 || H > 65535) return FG_ERR_BAD_SIZE;
    for (int d : {a_dtype, w_dtype, c_dtype})
        if (d != FG_F32 && d != FG_BF16) return FG_ERR_BAD_DTYPE;
    const int RM = M <= 8 ? 8 : HV_ROWS;
    if (M <= HV_ROWS && (size_t)RM * (K + 3) * sizeof(float) <= 48 * 1024) {
        const size_t rows = (size_t)RM * ((K + 3) / 4 * 4) * sizeof(float), sums = (size_t)4 * RM * HV_COLS * sizeof(float);
        const size_t smem = transposed && sums > rows ? sums : rows;
        const size_t es = w_dtype == FG_F32 ? 4 : 2;
        const int vec = transposed ? (N % 2 == 0 && ldw % 2 == 0 && ((uintptr_t)W % (2 * es)) == 0)
                                   : (K % (int)(16 / es) == 0 && ldw % (int)(16 / es) == 0 && ((uintptr_t)W & 15) == 0);
        const int cols = w_dtype == FG_F32 ? 4 * HV_COLS : HV_COLS;
        const dim3 grid(transposed ? (N + cols - 1) / cols : (N + 15) / 16, H);
#define HV_LAUNCH(TW, TR, R_) fg_launch(head_gemv_kernel<TW, TR, R_>, grid, dim3(256), smem, stream, A, a_dtype, lda, a_stride, (const TW *)W, ldw, C, \
                                        c_dtype, ldc, c_stride, gate, ldg, M, N, K, vec)
#define HV_BY_ROWS(TW, TR) (RM == 8 ? HV_LAUNCH(TW, TR, 8) : HV_LAUNCH(TW, TR, 16))
        if (w_dtype == FG_F32) return transposed ? HV_BY_ROWS(float, true) : HV_BY_ROWS(float, false);
        return transposed ? HV_BY_ROWS(bf16, true) : HV_BY_ROWS(bf16, false);
#undef HV_BY_ROWS
#undef HV_LAUNCH
    }
    dim3 grid((N + HG_T - 1) / HG_T, (M + HG_T - 1) / HG_T, H);
    if (grid.y > 65535) return FG_ERR_BAD_SIZE;
    return fg_launch(head_gemm_kernel, grid, dim3(256), 0, stream, A, a_dtype, lda, a_stride, W, w_dtype, ldw, transposed, C, c_dtype, ldc, c_stride,
                     gate, ldg, M, N, K);
}
