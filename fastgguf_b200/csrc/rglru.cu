// The real-gated linear recurrent unit and what stands between its projections and its output projection.
//
// A recurrent block has two branches of C channels, y and x (both out of one contraction, float32, without their biases):
//     u = conv_b + causal convolution over time per channel of (x + x_bias)      weights [taps][C], the last for the
//                                                                                token itself; zeros before the sequence
//     r = sigmoid(R u + r_bias), i = sigmoid(I u + i_bias)                       R, I block diagonal: `blocks` squares of C / blocks
//     log a = -gain r softplus(lam);  S_t = a S_(t-1) + sqrt(1 - a^2) i u;       out = S gelu_tanh(y + y_bias)
// Everything here is 32-bit in every engine dtype; only out takes the engine's.
//
// State row of a sequence: [a ring of `taps` convolution inputs, each C floats (none with one tap) | S, C floats].  The input of
// position p lies at p mod taps, so a single-token step reads the entries of p - 1 .. p - taps + 1 and writes that of p, which is
// none of them: one kernel does both, whatever order its blocks run in.
//
//   fg_rglru_step: a step of single tokens, all of it in ONE launch - a block per (16 channels of a part, 8 rows) forms u of the
//     whole part in shared memory, its warps stream two channels' rows of R and I for the eight rows, and the lanes that end up
//     with a (channel, row) finish it.
//   fg_rglru_conv, the gates, fg_rglru_scan: prompts and portions.  The gates' contraction reads u in 32 bits; so that the tensor
//     cores can run it, fg_rglru_conv also writes u as three bfloat16 numbers whose sum is u (8 + 8 + 8 bits of mantissa): with
//     the matrix three times side by side along k, products of bfloat16 numbers are exact and the sum is a 32-bit one.
//   fg_rglru_scan: the recurrence is linear with a diagonal matrix, so it is cut along time: a thread owns a channel and
//     SCAN_T tokens, forms their (a, b) once in registers and composes them; the compositions of a block's warps meet in shared
//     memory, those of a cluster's blocks in one another's, and every thread then walks its tokens from the right start.
#include "common.cuh"

#define SCAN_W 8                      // warps a block (a warp: 32 channels)
#define SCAN_T 16                     // tokens a thread
#define SCAN_MAX_CLUSTER 8
#define STEP_ROWS 8                   // rows (sequences) a block of the single-token kernel serves
#define STEP_CHANNELS 16              // channels it finishes, two a warp
#define CONV_ROWS 8                   // rows a thread of the convolution takes

// exponential, division and square root on the special-function unit (each within 2 ulp, the exponential's argument rounded once)
__device__ __forceinline__ float rg_sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float rg_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float rg_gelu(float z) { return z * rg_sigmoid(1.5957691216f * fmaf(0.044715f * z * z, z, z)); }   // 0.5 (1 + tanh(y)) = sigmoid(2 y)
__device__ __forceinline__ float rg_sqrt(float x) {
    float r;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
// a and the input term of one token: rate = gain * softplus(lam)
__device__ __forceinline__ void rg_coefficients(float zr, float zi, float u, float rate, float &a, float &b) {
    const float log_a = -rate * rg_sigmoid(zr);
    a = __expf(log_a);
    // 1 - a^2 = 1 - e^x, x = 2 log a <= 0: where a is close to one the series -x (1 + x/2 + x^2/6 + ...), so that nothing cancels
    // (|x| < 1/4: the first term left out is below 2e-8 of the sum), else the difference
    const float x = 2.0f * log_a;
    float p = fmaf(x, 1.0f / 5040.0f, 1.0f / 720.0f);
    p = fmaf(x, p, 1.0f / 120.0f);
    p = fmaf(x, p, 1.0f / 24.0f);
    p = fmaf(x, p, 1.0f / 6.0f);
    p = fmaf(x, p, 0.5f);
    p = fmaf(x, p, 1.0f);
    const float rest = x > -0.25f ? -x * p : fmaf(-a, a, 1.0f);
    b = rg_sqrt(rest) * (rg_sigmoid(zi) * u);
}

// ------------------------------------------------------------------ convolution, prompts and portions
// NC neighbouring channels (1 or 4) and CONV_ROWS rows a thread; TAPS > 0: that many, 0: `taps`.  Rows whose taps all lie in this
// step are the common case: a thread's inputs are then fetched once, together.  pieces (optional): [part][row][3][size of a
// part] bfloat16, see above.  tiles (optional): the table of the grouped contraction that reads them - for each part, for each tile
// along its outputs, its rows in runs of 128.
template <int NC> struct RgVec { float v[NC]; };
template <int NC> __device__ __forceinline__ RgVec<NC> rg_load(const float *p) {
    RgVec<NC> r;
    if (NC == 4) { const float4 t = *(const float4 *)p; r.v[0] = t.x; r.v[NC > 1 ? 1 : 0] = t.y; r.v[NC > 2 ? 2 : 0] = t.z; r.v[NC > 3 ? 3 : 0] = t.w; }
    else r.v[0] = *p;
    return r;
}
template <int NC> __device__ __forceinline__ void rg_store_conv(const RgVec<NC> &acc, float *u, bf16 *dst, int part) {
    if (NC == 4) *(float4 *)u = make_float4(acc.v[0], acc.v[NC > 1 ? 1 : 0], acc.v[NC > 2 ? 2 : 0], acc.v[NC > 3 ? 3 : 0]);
    else *u = acc.v[0];
    if (!dst) return;
    float rest[NC];
#pragma unroll
    for (int q = 0; q < NC; q++) rest[q] = acc.v[q];
#pragma unroll
    for (int e = 0; e < 3; e++, dst += part) {
        __align__(8) bf16 h[NC];
#pragma unroll
        for (int q = 0; q < NC; q++) { h[q] = __float2bfloat16_rn(rest[q]); rest[q] -= __bfloat162float(h[q]); }
        if (NC == 4) *(uint2 *)dst = *(const uint2 *)h;
        else dst[0] = h[0];
    }
}

template <int NC, int TAPS>
__global__ void __launch_bounds__(256)
rglru_conv_kernel(const float *__restrict__ x, int ld, const float *__restrict__ x_bias, const float *__restrict__ w,
                  const float *__restrict__ conv_b, int taps_, const float *__restrict__ state, long long state_stride,
                  const int *__restrict__ positions, const int *__restrict__ row_seq, const int *__restrict__ cu_rows,
                  const int *__restrict__ slots, float *__restrict__ u, int ldu, bf16 *__restrict__ pieces, int4 *__restrict__ tiles,
                  int n_tiles, int tiles_n, int M, int C, int part) {
    pdl_wait();
    if (tiles && blockIdx.x == 0 && blockIdx.y == 0) {
        const int row_tiles = (M + 127) / 128;
        for (int t = threadIdx.x; t < n_tiles; t += 256) {
            const int b = t / (tiles_n * row_tiles), rest = t - b * tiles_n * row_tiles, qt = rest / row_tiles, rt = rest - qt * row_tiles;
            tiles[t] = make_int4(b * M + rt * 128, (b + 1) * M, b * 2 * part, qt);
        }
    }
    const int taps = TAPS > 0 ? TAPS : taps_;
    const int c = (blockIdx.y * 256 + threadIdx.x) * NC;
    if (c >= C) return;
    const RgVec<NC> xb = rg_load<NC>(x_bias + c), cb = rg_load<NC>(conv_b + c);
    const int p = c / part, j0 = c - p * part;               // (a part is a multiple of NC)
    const int m0 = blockIdx.x * CONV_ROWS, m1 = min(M, m0 + CONV_ROWS);
    bf16 *dst0 = pieces ? pieces + ((size_t)p * M) * 3 * part + j0 : nullptr;
    if (TAPS > 0 && m1 - m0 == CONV_ROWS) {
        const int s = row_seq[m0];
        if (cu_rows[s] + TAPS - 1 <= m0 && row_seq[m1 - 1] == s) {
            RgVec<NC> in[CONV_ROWS + (TAPS > 0 ? TAPS : 1) - 1], wt[TAPS > 0 ? TAPS : 1];
#pragma unroll
            for (int i = 0; i < CONV_ROWS + TAPS - 1; i++) in[i] = rg_load<NC>(x + (size_t)(m0 - (TAPS - 1) + i) * ld + c);
#pragma unroll
            for (int t = 0; t < TAPS; t++) wt[t] = rg_load<NC>(w + (size_t)t * C + c);
#pragma unroll
            for (int i = 0; i < CONV_ROWS + TAPS - 1; i++)
#pragma unroll
                for (int q = 0; q < NC; q++) in[i].v[q] += xb.v[q];
#pragma unroll
            for (int i = 0; i < CONV_ROWS; i++) {
                RgVec<NC> acc = cb;
#pragma unroll
                for (int t = 0; t < TAPS; t++)
#pragma unroll
                    for (int q = 0; q < NC; q++) acc.v[q] = fmaf(wt[t].v[q], in[i + t].v[q], acc.v[q]);
                rg_store_conv<NC>(acc, u + (size_t)(m0 + i) * ldu + c, dst0 ? dst0 + (size_t)(m0 + i) * 3 * part : nullptr, part);
            }
            return;
        }
    }
    for (int m = m0; m < m1; m++) {
        const int s = row_seq[m], i = m - cu_rows[s], pos = positions[m];
        const float *ring = state + (size_t)slots[s] * state_stride;
        RgVec<NC> acc = cb;
        for (int back = taps - 1; back >= 0; back--) {
            RgVec<NC> v;
            if (back <= i) {
                v = rg_load<NC>(x + (size_t)(m - back) * ld + c);
#pragma unroll
                for (int q = 0; q < NC; q++) v.v[q] += xb.v[q];
            } else if (pos - back >= 0) v = rg_load<NC>(ring + (size_t)((pos - back) % taps) * C + c);
            else continue;
            const RgVec<NC> wt = rg_load<NC>(w + (size_t)(taps - 1 - back) * C + c);
#pragma unroll
            for (int q = 0; q < NC; q++) acc.v[q] = fmaf(wt.v[q], v.v[q], acc.v[q]);
        }
        rg_store_conv<NC>(acc, u + (size_t)m * ldu + c, dst0 ? dst0 + (size_t)m * 3 * part : nullptr, part);
    }
}

// ------------------------------------------------------------------ the recurrence over a portion
__device__ __forceinline__ void rg_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float rg_remote(const float *p, int rank) {
    const uint32_t local = (uint32_t)__cvta_generic_to_shared(p);
    uint32_t remote;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}

// z: the gates' raw numbers, row m of part p at z + m * z_row + p * z_part: [r: part | i: part]; gate_bias the same for one row.
// grid (channel tiles of 32, sequences, blocks of the cluster): the cluster's blocks stand one after another along time.
template <typename TO>
__global__ void __launch_bounds__(SCAN_W * 32)
rglru_scan_kernel(const float *__restrict__ z, int z_row, long long z_part, const float *__restrict__ gate_bias,
                  const float *__restrict__ u, int ldu, const float *__restrict__ lam, float gain, const float *__restrict__ proj, int ldp,
                  const float *__restrict__ proj_bias, TO *__restrict__ out, int ldo, const int *__restrict__ cu_rows,
                  const int *__restrict__ slots, const int *__restrict__ positions, float *__restrict__ state, long long state_stride, int C,
                  int part, int taps) {
    __shared__ float agg_a[SCAN_W][32], agg_b[SCAN_W][32];
    __shared__ float tot_a[2][32], tot_b[2][32];
    pdl_wait();
    const int seq = blockIdx.y, rank = blockIdx.z, CS = gridDim.z, warp = warp_index(), lane = threadIdx.x & 31;
    const int row0 = cu_rows[seq], row1 = cu_rows[seq + 1];
    if (row1 <= row0) return;                                   // the whole cluster leaves
    const int c = blockIdx.x * 32 + lane;
    const bool live = c < C;
    const int cc = live ? c : 0, p = cc / part, j = cc - p * part;
    const float *zr = z + p * z_part + j, *zi = zr + part;
    const float br = gate_bias[(size_t)p * 2 * part + j], bi = gate_bias[(size_t)p * 2 * part + part + j];
    const float rate = gain * rg_softplus(lam[cc]), yb = proj_bias[cc];
    float *ring = state + (size_t)slots[seq] * state_stride, *Sg = ring + (taps > 1 ? (size_t)taps * C : 0);
    float carry = live ? Sg[c] : 0.f;
    int it = 0;
    for (int t0 = row0; t0 < row1; t0 += CS * SCAN_W * SCAN_T, it ^= 1) {
        const int first = t0 + (rank * SCAN_W + warp) * SCAN_T;
        const int n = live ? max(0, min(SCAN_T, row1 - first)) : 0;
        const bool full = __all_sync(0xffffffffu, n == SCAN_T);        // the common case has no predicates
        float a[SCAN_T], b[SCAN_T], y[SCAN_T];
        {
            float vr[SCAN_T], vi[SCAN_T], vu[SCAN_T];            // all loads on their way before the first is used
            const float *zrp = zr + (size_t)first * z_row, *zip = zi + (size_t)first * z_row, *up = u + (size_t)first * ldu + cc,
                        *yp = proj + (size_t)first * ldp + cc;
            if (full) {
#pragma unroll
                for (int i = 0; i < SCAN_T; i++) { vr[i] = zrp[i * z_row]; vi[i] = zip[i * z_row]; vu[i] = up[i * ldu]; }
#pragma unroll
                for (int i = 0; i < SCAN_T; i++) y[i] = yp[i * ldp];
#pragma unroll
                for (int i = 0; i < SCAN_T; i++) rg_coefficients(vr[i] + br, vi[i] + bi, vu[i], rate, a[i], b[i]);
            } else {
#pragma unroll
                for (int i = 0; i < SCAN_T; i++) {
                    vr[i] = i < n ? zrp[i * z_row] : 0.f;
                    vi[i] = i < n ? zip[i * z_row] : 0.f;
                    vu[i] = i < n ? up[i * ldu] : 0.f;
                    y[i] = i < n ? yp[i * ldp] : 0.f;
                }
#pragma unroll
                for (int i = 0; i < SCAN_T; i++) {
                    rg_coefficients(vr[i] + br, vi[i] + bi, vu[i], rate, a[i], b[i]);
                    if (i >= n) { a[i] = 1.f; b[i] = 0.f; }
                }
            }
        }
        float wa = 1.f, wb = 0.f;                               // this thread's tokens composed: S -> wa S + wb
#pragma unroll
        for (int i = 0; i < SCAN_T; i++) { wb = fmaf(a[i], wb, b[i]); wa *= a[i]; }
        agg_a[warp][lane] = wa;
        agg_b[warp][lane] = wb;
        __syncthreads();
        float pa = 1.f, pb = 0.f, ta = 1.f, tb = 0.f;           // before this warp; the whole block
#pragma unroll
        for (int w = 0; w < SCAN_W; w++) {
            if (w == warp) { pa = ta; pb = tb; }
            tb = fmaf(agg_a[w][lane], tb, agg_b[w][lane]);
            ta *= agg_a[w][lane];
        }
        float start = carry;
        if (CS > 1) {
            if (warp == 0) { tot_a[it][lane] = ta; tot_b[it][lane] = tb; }
            rg_cluster_sync();                                  // (two sets of totals: the next but one iteration's writes come after everybody's reads)
            float S = carry, ra[SCAN_MAX_CLUSTER], rb[SCAN_MAX_CLUSTER];
#pragma unroll
            for (int r = 0; r < SCAN_MAX_CLUSTER; r++) {
                ra[r] = r < CS ? rg_remote(&tot_a[it][lane], r) : 1.f;
                rb[r] = r < CS ? rg_remote(&tot_b[it][lane], r) : 0.f;
            }
#pragma unroll
            for (int r = 0; r < SCAN_MAX_CLUSTER; r++) {
                if (r == rank) start = S;
                S = fmaf(ra[r], S, rb[r]);
            }
            carry = S;
        } else {
            carry = fmaf(ta, carry, tb);
            __syncthreads();                                    // the compositions are read before the next ones are written
        }
        float S = fmaf(pa, start, pb);
        TO *op = out + (size_t)first * ldo + cc;
        if (full) {
#pragma unroll
            for (int i = 0; i < SCAN_T; i++) {
                S = fmaf(a[i], S, b[i]);
                op[i * ldo] = from_f32<TO>(S * rg_gelu(y[i] + yb));
            }
        } else {
#pragma unroll
            for (int i = 0; i < SCAN_T; i++) {
                S = fmaf(a[i], S, b[i]);
                if (i < n) op[i * ldo] = from_f32<TO>(S * rg_gelu(y[i] + yb));
            }
        }
    }
    if (CS > 1) rg_cluster_sync();                              // nobody's totals go away while they are being read
    if (rank != 0 || !live) return;
    if (warp == 0) Sg[c] = carry;
    else if (warp == 1 && taps > 1) {
        // the portion's last inputs of the convolution to their places in the ring
        const float xb = proj_bias[C + c];
        const int n = row1 - row0, pos0 = positions[row0];
        for (int i = max(0, n - (taps - 1)); i < n; i++) ring[(size_t)((pos0 + i) % taps) * C + c] = proj[(size_t)(row0 + i) * ldp + C + c] + xb;
    }
}

// ------------------------------------------------------------------ a step of single tokens
// W: [part][2 * size][size] rows of R, then of I.  grid (16 channels of a part, parts, 8 rows).
template <typename TW, typename TO>
__global__ void __launch_bounds__(256)
rglru_step_kernel(const float *__restrict__ proj, int ldp, const float *__restrict__ proj_bias, const float *__restrict__ conv_w,
                  const float *__restrict__ conv_b, int taps, const TW *__restrict__ W, const float *__restrict__ gate_bias,
                  const float *__restrict__ lam, float gain, const int *__restrict__ positions, const int *__restrict__ row_seq,
                  const int *__restrict__ slots, float *__restrict__ state, long long state_stride, TO *__restrict__ out, int ldo, int M, int C,
                  int part, int stride, int vec, int vec4) {
    extern __shared__ __align__(16) float us[];                 // [STEP_ROWS][stride] u of the part
    constexpr int VEC = 16 / (int)sizeof(TW);
    const int p = blockIdx.y, warp = warp_index(), lane = threadIdx.x & 31;
    const int j0 = blockIdx.x * STEP_CHANNELS + warp * 2;       // the warp's channels j0, j0 + 1 of the part
    // the warp's four rows: R of both channels, then I of both (channels beyond the part repeat its last one and are not stored)
    const TW *wr[4];
#pragma unroll
    for (int q = 0; q < 4; q++) wr[q] = W + ((size_t)p * 2 * part + (q >> 1) * part + min(j0 + (q & 1), part - 1)) * part;
    uint4 w4[4];
    const bool have = vec && lane * VEC < part;
    if (have) {                                                  // weights: before the wait on the contraction in front
#pragma unroll
        for (int q = 0; q < 4; q++) w4[q] = *(const uint4 *)(wr[q] + lane * VEC);
    }
    // what the lanes that finish a (channel, row) need besides the sums: asked for early, used at the end
    const int jf = j0 + ((lane >> 3) & 1), mf = blockIdx.z * STEP_ROWS + (lane & 7), cf = p * part + min(jf, part - 1);
    const bool finish = lane < 16 && jf < part && mf < M;
    const float br = gate_bias[(size_t)p * 2 * part + min(jf, part - 1)], bi = gate_bias[(size_t)p * 2 * part + part + min(jf, part - 1)];
    const float lam_c = lam[cf], yb = proj_bias[cf];
    pdl_launch_dependents_small_step(M);
    pdl_wait();
    float *Sg = nullptr;
    float S0 = 0.f, y0 = 0.f;
    if (finish) {
        y0 = proj[(size_t)mf * ldp + cf];
        Sg = state + (size_t)slots[row_seq[mf]] * state_stride + (taps > 1 ? (size_t)taps * C : 0) + cf;
        S0 = *Sg;
    }
    {
        // u of the part: warp w the row m0 + w, its lanes NC channels at a time
        const int m = blockIdx.z * STEP_ROWS + warp;
        float *urow = us + warp * stride;
        if (m < M) {
            const int pos = positions[m];
            float *ring = state + (size_t)slots[row_seq[m]] * state_stride;
            const float *now = proj + (size_t)m * ldp + C;
            if (vec4) {
                for (int j = lane * 4; j < part; j += 128) {
                    const int c = p * part + j;
                    RgVec<4> acc = rg_load<4>(conv_b + c), cur = rg_load<4>(now + c);
                    const RgVec<4> xb = rg_load<4>(proj_bias + C + c), wl = rg_load<4>(conv_w + (size_t)(taps - 1) * C + c);
#pragma unroll
                    for (int q = 0; q < 4; q++) cur.v[q] += xb.v[q];
#pragma unroll 4
                    for (int back = 1; back < taps; back++) {
                        if (pos - back < 0) break;
                        const RgVec<4> old = rg_load<4>(ring + (size_t)((pos - back) % taps) * C + c), wt = rg_load<4>(conv_w + (size_t)(taps - 1 - back) * C + c);
#pragma unroll
                        for (int q = 0; q < 4; q++) acc.v[q] = fmaf(wt.v[q], old.v[q], acc.v[q]);
                    }
#pragma unroll
                    for (int q = 0; q < 4; q++) acc.v[q] = fmaf(wl.v[q], cur.v[q], acc.v[q]);
                    *(float4 *)(urow + j) = make_float4(acc.v[0], acc.v[1], acc.v[2], acc.v[3]);
                    if (taps > 1 && j / STEP_CHANNELS == blockIdx.x)
                        *(float4 *)(ring + (size_t)(pos % taps) * C + c) = make_float4(cur.v[0], cur.v[1], cur.v[2], cur.v[3]);
                }
            } else {
                for (int j = lane; j < part; j += 32) {
                    const int c = p * part + j;
                    const float cur = now[c] + proj_bias[C + c];
                    float acc = conv_b[c];
                    for (int back = 1; back < taps; back++)
                        if (pos - back >= 0) acc = fmaf(conv_w[(size_t)(taps - 1 - back) * C + c], ring[(size_t)((pos - back) % taps) * C + c], acc);
                    urow[j] = fmaf(conv_w[(size_t)(taps - 1) * C + c], cur, acc);
                    if (taps > 1 && j / STEP_CHANNELS == blockIdx.x) ring[(size_t)(pos % taps) * C + c] = cur;
                }
            }
        } else {
            for (int j = lane; j < part; j += 32) urow[j] = 0.f;
        }
    }
    __syncthreads();
    float v[4 * STEP_ROWS];                                      // [row of W][row of the step]
#pragma unroll
    for (int i = 0; i < 4 * STEP_ROWS; i++) v[i] = 0.f;
    if (vec) {
        for (int k = lane * VEC; k < part; k += 32 * VEC) {
#pragma unroll
            for (int q = 0; q < 4; q++)
                if (k >= 32 * VEC) w4[q] = *(const uint4 *)(wr[q] + k);
#pragma unroll
            for (int row = 0; row < STEP_ROWS; row++) {
                float x[VEC];
#pragma unroll
                for (int i = 0; i < VEC; i += 4) *(float4 *)(x + i) = *(const float4 *)(us + row * stride + k + i);
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    const TW *we = (const TW *)&w4[q];
#pragma unroll
                    for (int i = 0; i < VEC; i++) v[q * STEP_ROWS + row] = fmaf(x[i], to_f32<TW>(we[i]), v[q * STEP_ROWS + row]);
                }
            }
        }
    } else {
        for (int k = lane; k < part; k += 32) {
            float w[4];
#pragma unroll
            for (int q = 0; q < 4; q++) w[q] = to_f32<TW>(wr[q][k]);
#pragma unroll
            for (int row = 0; row < STEP_ROWS; row++) {
                const float x = us[row * stride + k];
#pragma unroll
                for (int q = 0; q < 4; q++) v[q * STEP_ROWS + row] = fmaf(x, w[q], v[q * STEP_ROWS + row]);
            }
        }
    }
    // 32 sums over 32 lanes: at every exchange a lane keeps half of its numbers, and ends with sum number `lane`
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < o; i++) {
            const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
    const float zi = __shfl_xor_sync(0xffffffffu, v[0], 16);     // lanes 0 .. 15: R u of (channel lane / 8, row lane % 8); I u from lane + 16
    if (!finish) return;
    float a, b;
    rg_coefficients(v[0] + br, zi + bi, us[(lane & 7) * stride + jf], gain * rg_softplus(lam_c), a, b);
    const float S = fmaf(a, S0, b);
    *Sg = S;
    out[(size_t)mf * ldo + cf] = from_f32<TO>(S * rg_gelu(y0 + yb));
}

// ------------------------------------------------------------------ launchers
// floats of a sequence's state row
extern "C" long long fg_rglru_state_floats(int C, int taps) { return (long long)(taps > 1 ? taps + 1 : 1) * C; }

// proj: [M, ldp] float32, columns [y: C | x: C] without their biases (proj_bias [2 C]); u: [M, ldu] float32.  pieces (or null):
// [C / part][M][3 * part] bfloat16, tiles (with pieces): the grouped contraction's table for outputs of 2 * part in tiles of bn,
// fg_rglru_tiles(M, C, part, bn) entries.
extern "C" int fg_rglru_tiles(int M, int C, int part, int bn) { return (C / part) * ((2 * part + bn - 1) / bn) * ((M + 127) / 128); }

extern "C" int fg_rglru_conv(const float *proj, int ldp, const float *proj_bias, const float *conv_w, const float *conv_b, int taps,
                             const float *state, long long state_stride, const int *positions, const int *row_seq, const int *cu_rows,
                             const int *slots, float *u, int ldu, void *pieces, void *tiles, int bn, int M, int C, int part, cudaStream_t stream) {
    if (M <= 0) return 0;
    if (C <= 0 || part <= 0 || C % part || taps <= 0 || (pieces && (!tiles || bn <= 0))) return FG_ERR_BAD_SIZE;
    const bool four = part % 4 == 0 && ldp % 4 == 0 && ldu % 4 == 0 &&
                      ((((uintptr_t)proj) | ((uintptr_t)proj_bias) | ((uintptr_t)conv_w) | ((uintptr_t)conv_b) | ((uintptr_t)u)) & 15) == 0 &&
                      (((uintptr_t)pieces) & 7) == 0 && (((uintptr_t)state) & 15) == 0 && state_stride % 4 == 0;
    const int n_tiles = pieces ? fg_rglru_tiles(M, C, part, bn) : 0, tiles_n = pieces ? (2 * part + bn - 1) / bn : 0;
    const int per = four ? 1024 : 256;
    const dim3 grid((M + CONV_ROWS - 1) / CONV_ROWS, (C + per - 1) / per);
#define RG_CONV(NC, TAPS) fg_launch(rglru_conv_kernel<NC, TAPS>, grid, dim3(256), 0, stream, proj + C, ldp, proj_bias + C, conv_w, conv_b, taps, state, \
                                    state_stride, positions, row_seq, cu_rows, slots, u, ldu, (bf16 *)pieces, (int4 *)tiles, n_tiles, tiles_n, M, C, part)
    if (!four) return RG_CONV(1, 0);
    switch (taps) {
    case 2: return RG_CONV(4, 2);
    case 3: return RG_CONV(4, 3);
    case 4: return RG_CONV(4, 4);
    default: return RG_CONV(4, 0);
    }
#undef RG_CONV
}

// z: the gates' raw numbers (row m of part p: [r | i] at z + m * z_row + p * z_part); gate_bias: [C / part][2 * part]; lam: [C];
// out: [M, ldo] in out_dtype.  Brings the state rows up to date.  max_new: the longest portion of the step.
extern "C" int fg_rglru_scan(const float *z, int z_row, long long z_part, const float *gate_bias, const float *u, int ldu,
                             const float *lam, float gain, const float *proj, int ldp, const float *proj_bias, void *out, int out_dtype, int ldo,
                             const int *cu_rows, const int *slots, const int *positions, float *state, long long state_stride, int n_seq,
                             int max_new, int C, int part, int taps, cudaStream_t stream) {
    if (n_seq <= 0 || max_new <= 0) return 0;
    if (C <= 0 || part <= 0 || C % part || taps <= 0 || n_seq > 65535) return FG_ERR_BAD_SIZE;
    int cs = 1;
    while (cs < SCAN_MAX_CLUSTER && cs * SCAN_W * SCAN_T < max_new) cs *= 2;
    const dim3 grid((C + 31) / 32, n_seq, cs);
    if (out_dtype == FG_F32)
        return fg_launch_cluster(rglru_scan_kernel<float>, grid, dim3(SCAN_W * 32), 0, stream, cs, z, z_row, z_part, gate_bias, u, ldu, lam, gain, proj,
                                 ldp, proj_bias, (float *)out, ldo, cu_rows, slots, positions, state, state_stride, C, part, taps);
    if (out_dtype == FG_BF16)
        return fg_launch_cluster(rglru_scan_kernel<bf16>, grid, dim3(SCAN_W * 32), 0, stream, cs, z, z_row, z_part, gate_bias, u, ldu, lam, gain, proj,
                                 ldp, proj_bias, (bf16 *)out, ldo, cu_rows, slots, positions, state, state_stride, C, part, taps);
    return FG_ERR_BAD_DTYPE;
}

// 1 if the single-token kernel holds a part of this size in shared memory
extern "C" int fg_rglru_step_ok(int part) { return part > 0 && (size_t)STEP_ROWS * ((part + 3) / 4 * 4) * sizeof(float) <= 200 * 1024; }

template <typename TW, typename TO>
static int rglru_step_launch(const float *proj, int ldp, const float *proj_bias, const float *conv_w, const float *conv_b, int taps, const void *W,
                             const float *gate_bias, const float *lam, float gain, const int *positions, const int *row_seq, const int *slots,
                             float *state, long long state_stride, void *out, int ldo, int M, int C, int part, cudaStream_t stream) {
    static FgPerDevice setup;
    if (fg_needs_setup(setup)) {
        cudaError_t e = cudaFuncSetAttribute(rglru_step_kernel<TW, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return (int)e;
    }
    const int stride = (part + 3) / 4 * 4, vec = part % (16 / (int)sizeof(TW)) == 0 && (((uintptr_t)W) & 15) == 0;
    const int vec4 = part % 4 == 0 && ldp % 4 == 0 && state_stride % 4 == 0 &&
                     ((((uintptr_t)proj) | ((uintptr_t)proj_bias) | ((uintptr_t)conv_w) | ((uintptr_t)conv_b) | ((uintptr_t)state)) & 15) == 0;
    const dim3 grid((part + STEP_CHANNELS - 1) / STEP_CHANNELS, C / part, (M + STEP_ROWS - 1) / STEP_ROWS);
    return fg_launch(rglru_step_kernel<TW, TO>, grid, dim3(256), (size_t)STEP_ROWS * stride * sizeof(float), stream, proj, ldp, proj_bias, conv_w,
                     conv_b, taps, (const TW *)W, gate_bias, lam, gain, positions, row_seq, slots, state, state_stride, (TO *)out, ldo, M, C, part, stride, vec, vec4);
}

// A step of single tokens (one row a sequence).  W: [C / part][2 * part][part] in w_dtype.
extern "C" int fg_rglru_step(const float *proj, int ldp, const float *proj_bias, const float *conv_w, const float *conv_b, int taps,
                             const void *W, int w_dtype, const float *gate_bias, const float *lam, float gain, const int *positions,
                             const int *row_seq, const int *slots, float *state, long long state_stride, void *out, int out_dtype, int ldo, int M,
                             int C, int part, cudaStream_t stream) {
    if (M <= 0) return 0;
    if (C <= 0 || part <= 0 || C % part || taps <= 0 || C / part > 65535 || M > 65535 * STEP_ROWS || !fg_rglru_step_ok(part)) return FG_ERR_BAD_SIZE;
#define RG_STEP(TW, TO) rglru_step_launch<TW, TO>(proj, ldp, proj_bias, conv_w, conv_b, taps, W, gate_bias, lam, gain, positions, row_seq, slots, state, \
                                                  state_stride, out, ldo, M, C, part, stream)
    if (w_dtype == FG_F32) return out_dtype == FG_F32 ? RG_STEP(float, float) : out_dtype == FG_BF16 ? RG_STEP(float, bf16) : FG_ERR_BAD_DTYPE;
    if (w_dtype == FG_BF16) return out_dtype == FG_F32 ? RG_STEP(bf16, float) : out_dtype == FG_BF16 ? RG_STEP(bf16, bf16) : FG_ERR_BAD_DTYPE;
#undef RG_STEP
    return FG_ERR_BAD_DTYPE;
}
