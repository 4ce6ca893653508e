// Linear attention with a fixed decay per head on bfloat16 activations: the tensor-core forms of what retention.cu computes on the
// FMA units for mixers whose q, k and v are activations of the engine's dtype (silu of a projection) and whose outputs are taken as
// they are (a norm over all heads and a gate follow).
//
//     S_t = decay S_(t-1) + k_t v_t^T (S: [dk, dv] float32),  o_t = S_t^T q_t
//
// A row of `proj` (bfloat16) holds q [H, dk] | k [H, dk] | v [H, dv] | g [H, dv]; q, k and v pass silu in float32 and are rounded to
// bfloat16 once.  Everything behind that is 32-bit: decays, scores times decays, state, outputs.  For the tensor cores a float32
// number (a key times its decay, a weighted score, an entry of the state) is written as three bfloat16 numbers that sum to it (8 + 8 + 8
// bits of mantissa); products of two bfloat16 numbers are exact in float32 and the sums are float32 sums, so nothing is rounded to
// bfloat16 on the way.
//
//   portions   chunks of DC tokens of all sequences and heads at once:
//       1. decay_state_kernel   U_c = sum_t (decay^(n-1-t) k_t) v_t^T; q, k and v become their activations in place
//       2. decay_scan_kernel    over a sequence's chunks: the state in front of chunk c, as three bfloat16 numbers an entry
//       3. decay_out_kernel     o_i = decay^(i+1) S^T q_i + sum_(j<=i) decay^(i-j) (q_i . k_j) v_j
//   single tokens and short portions   decay_step_kernel: the state in registers, a block per (sequence, head)
//   row_norm_gate_kernel   out = o / sqrt(mean(o^2) + eps) * w * gate(g) over a whole row
// Head sizes 64 and 128 (keys and values each).
#include "attention_mma.cuh"

#define DC 64                       // tokens a chunk
#define DA_THREADS 256

// (fast exponential and division, 2 ulp each: the result is rounded to bfloat16 right after)
__device__ __forceinline__ float da_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
// silu of a projection's bfloat16, rounded to bfloat16
__device__ __forceinline__ float da_act(bf16 z) { return __bfloat162float(__float2bfloat16_rn(da_silu(__bfloat162float(z)))); }

// x = hi + mid + lo, each bfloat16 (exact: 24 bits of mantissa in three runs of 8)
__device__ __forceinline__ void split3(float x, bf16 &hi, bf16 &mid, bf16 &lo) {
    hi = __float2bfloat16_rn(x);
    const float r = x - __bfloat162float(hi);
    mid = __float2bfloat16_rn(r);
    lo = __float2bfloat16_rn(r - __bfloat162float(mid));
}
__device__ __forceinline__ void split3_pair(float a, float b, uint32_t &hi, uint32_t &mid, uint32_t &lo) {
    __nv_bfloat162 h, m, l;
    split3(a, h.x, m.x, l.x);
    split3(b, h.y, m.y, l.y);
    hi = *(uint32_t *)&h; mid = *(uint32_t *)&m; lo = *(uint32_t *)&l;
}
// where a row's 16-byte piece lies in a swizzled tile (row pitch `pitch` bytes)
__device__ __forceinline__ uint8_t *tile_at(uint8_t *tile, int pitch, int row, int chunk) { return tile + row * pitch + ((chunk ^ (row & 7)) << 4); }
// eight activations at once
__device__ __forceinline__ uint4 act8(const uint4 &raw) {
    const bf16 *z = (const bf16 *)&raw;
    uint4 out;
    bf16 *o = (bf16 *)&out;
#pragma unroll
    for (int e = 0; e < 8; e++) o[e] = __float2bfloat16_rn(da_silu(__bfloat162float(z[e])));
    return out;
}

// 1. U[c, h] = sum_t (decay^(n-1-t) k_t) v_t^T: M = dk, N = dv, K = the chunk's tokens
template <int DK, int DV>
__global__ void __launch_bounds__(DA_THREADS, 2)
decay_state_kernel(bf16 *proj, int ld, const int *__restrict__ chunk_row, const int *__restrict__ chunk_len,
                   const float *__restrict__ decay, float *__restrict__ U, int H) {
    extern __shared__ __align__(128) uint8_t sm[];
    constexpr int KP = DK * 2, VP = DV * 2, PIECE = DC * KP;
    uint8_t *K0 = sm, *Vt = sm + 3 * PIECE;
    pdl_wait();                 // (no early release: in a step of many rows these kernels stand between tensor-memory contractions)
    const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = warp_index(), lane = tid & 31;
    const int r0 = chunk_row[c], n = chunk_len[c];
    const float l2 = log2f(decay[h]);
    // every load of the block is in flight before the first is used; the activations go back where the projections came from
    constexpr int NK = DC * (DK / 8) / DA_THREADS, NV = DC * (DV / 8) / DA_THREADS;
    bf16 *base = proj + (size_t)r0 * ld;
    uint4 q[NK], k[NK], v[NV];
#pragma unroll
    for (int i = 0; i < NK; i++) {
        const int e = tid + i * DA_THREADS, t = e / (DK / 8), ch = e % (DK / 8);
        const bf16 *src = base + (size_t)t * ld + (size_t)h * DK + ch * 8;
        k[i] = t < n ? *(const uint4 *)(src + (size_t)H * DK) : make_uint4(0, 0, 0, 0);
        q[i] = t < n ? *(const uint4 *)src : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int e = tid + i * DA_THREADS, t = e / (DV / 8), ch = e % (DV / 8);
        v[i] = t < n ? *(const uint4 *)(base + (size_t)t * ld + (size_t)2 * H * DK + (size_t)h * DV + ch * 8) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int i = 0; i < NK; i++) {
        const int e = tid + i * DA_THREADS, t = e / (DK / 8), ch = e % (DK / 8);
        const uint4 a = act8(k[i]);
        const bf16 *kk = (const bf16 *)&a;
        const float f = exp2f(l2 * (float)(n - 1 - t));
        uint4 piece[3];
#pragma unroll
        for (int j = 0; j < 4; j++)        // (rows behind the chunk's last token hold zeros)
            split3_pair(t < n ? __bfloat162float(kk[2 * j]) * f : 0.f, t < n ? __bfloat162float(kk[2 * j + 1]) * f : 0.f, ((uint32_t *)&piece[0])[j],
                        ((uint32_t *)&piece[1])[j], ((uint32_t *)&piece[2])[j]);
#pragma unroll
        for (int p = 0; p < 3; p++) *(uint4 *)tile_at(K0 + p * PIECE, KP, t, ch) = piece[p];
        if (t < n) {
            bf16 *dst = base + (size_t)t * ld + (size_t)h * DK + ch * 8;
            *(uint4 *)(dst + (size_t)H * DK) = a;
            *(uint4 *)dst = act8(q[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int e = tid + i * DA_THREADS, t = e / (DV / 8), ch = e % (DV / 8);
        const uint4 a = act8(v[i]);
        *(uint4 *)tile_at(Vt, VP, t, ch) = a;
        if (t < n) *(uint4 *)(base + (size_t)t * ld + (size_t)2 * H * DK + (size_t)h * DV + ch * 8) = a;
    }
    __syncthreads();
    // a warp owns 16 rows of U and NW columns
    constexpr int MW = DK / 16, NW = DV / (8 / MW);
    const int m0 = (warp % MW) * 16, n0 = (warp / MW) * NW;
    const int mi = lane >> 3, r = lane & 7;
    const uint32_t ks = smem_addr(K0), vs = smem_addr(Vt);
    float acc[NW / 8][4];
#pragma unroll
    for (int d = 0; d < NW / 8; d++) acc[d][0] = acc[d][1] = acc[d][2] = acc[d][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DC / 16; kk++) {
        uint32_t a[3][4];
        {
            // K' is stored token by token, so the rows of U come by transposed loads
            const int row = kk * 16 + (mi >> 1) * 8 + r, ch = m0 / 8 + (mi & 1);
#pragma unroll
            for (int p = 0; p < 3; p++) ldmatrix_x4_trans(ks + p * PIECE + row * KP + ((ch ^ (row & 7)) << 4), a[p][0], a[p][1], a[p][2], a[p][3]);
        }
#pragma unroll
        for (int dd = 0; dd < NW / 16; dd++) {
            const int row = kk * 16 + (mi & 1) * 8 + r, ch = n0 / 8 + dd * 2 + (mi >> 1);
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(vs + row * VP + ((ch ^ (row & 7)) << 4), b0, b1, b2, b3);
#pragma unroll
            for (int p = 2; p >= 0; p--) {
                mma_bf16(acc[2 * dd], a[p], b0, b1);
                mma_bf16(acc[2 * dd + 1], a[p], b2, b3);
            }
        }
    }
    float *Ug = U + ((size_t)c * H + h) * DK * DV + (size_t)(m0 + (lane >> 2)) * DV + n0 + 2 * (lane & 3);
#pragma unroll
    for (int d = 0; d < NW / 8; d++) {
        *(float2 *)(Ug + d * 8) = make_float2(acc[d][0], acc[d][1]);
        *(float2 *)(Ug + 8 * DV + d * 8) = make_float2(acc[d][2], acc[d][3]);
    }
}

// 2. The scan over a sequence's chunks, four entries of the state a thread: P[c, h] = the state in front of chunk c as three bfloat16
// numbers an entry ([piece][dk * dv]); the state behind the last chunk goes back to the sequence's row.
__global__ void __launch_bounds__(DA_THREADS)
decay_scan_kernel(const int *__restrict__ seq_chunk0, const int *__restrict__ chunk_len, const int *__restrict__ slots, const float *__restrict__ decay,
                  const float *__restrict__ U, bf16 *__restrict__ P, float *__restrict__ state, int H, int size) {
    pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, e = (blockIdx.z * DA_THREADS + threadIdx.x) * 4;
    if (e >= size) return;
    const int c0 = seq_chunk0[seq], c1 = seq_chunk0[seq + 1];
    if (c1 <= c0) return;
    float4 *Sg = (float4 *)(state + ((size_t)slots[seq] * H + h) * size + e);
    const float l2 = log2f(decay[h]);
    float4 s = *Sg;
    const size_t step = (size_t)H * size;
    const float *u = U + ((size_t)c0 * H + h) * size + e;
    bf16 *dst = P + ((size_t)c0 * H + h) * 3 * size + e;
    for (int c = c0; c < c1; c += 8) {
        // eight chunks' contributions are fetched before the first is used: the chain of sums does not wait for memory
        float4 add[8];
        float f[8];
#pragma unroll
        for (int i = 0; i < 8; i++) {
            if (c + i < c1) add[i] = *(const float4 *)(u + (size_t)i * step);
            f[i] = c + i < c1 ? exp2f(l2 * (float)chunk_len[c + i]) : 1.f;
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            if (c + i >= c1) break;
            uint2 p0, p1, p2;
            split3_pair(s.x, s.y, p0.x, p1.x, p2.x);
            split3_pair(s.z, s.w, p0.y, p1.y, p2.y);
            *(uint2 *)dst = p0;
            *(uint2 *)(dst + size) = p1;
            *(uint2 *)(dst + 2 * size) = p2;
            dst += 3 * step;
            s.x = fmaf(s.x, f[i], add[i].x); s.y = fmaf(s.y, f[i], add[i].y); s.z = fmaf(s.z, f[i], add[i].z); s.w = fmaf(s.w, f[i], add[i].w);
        }
        u += 8 * step;
    }
    *Sg = s;
}

// 3. Outputs of a chunk, 64 value columns a block: warp w owns tokens 16 w .. 16 w + 15.  q goes from memory to the operand registers;
// keys, values and the state's pieces arrive by asynchronous copies, all in flight at once.
template <int DK, int DV>
__global__ void __launch_bounds__(128, 3)
decay_out_kernel(const bf16 *__restrict__ proj, int ld, float *__restrict__ out, int ldo, const int *__restrict__ chunk_row,
                 const int *__restrict__ chunk_len, const float *__restrict__ decay, const bf16 *__restrict__ P, int H) {
    extern __shared__ __align__(128) uint8_t sm[];
    constexpr int KP = DK * 2, NB = 64, VP = NB * 2, SPIECE = DK * VP;
    const uint32_t ks = smem_addr(sm), vs = ks + DC * KP, ss = vs + DC * VP;
    pdl_wait();                 // (no early release: in a step of many rows these kernels stand between tensor-memory contractions)
    const int c = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * NB, tid = threadIdx.x, warp = warp_index(), lane = tid & 31;
    const int r0 = chunk_row[c], n = chunk_len[c];
    const bf16 *base = proj + (size_t)r0 * ld, *S = P + ((size_t)c * H + h) * 3 * DK * DV + col0;
    auto at = [](uint32_t tile, int pitch, int row, int ch) { return tile + row * pitch + ((ch ^ (row & 7)) << 4); };
    // (rows behind the chunk's last token repeat it: their weights are zero, and their own outputs are not stored)
#pragma unroll
    for (int i = 0; i < DC * (DK / 8) / 128; i++) {
        const int e = tid + i * 128, t = e / (DK / 8), ch = e % (DK / 8);
        cp_async16(at(ks, KP, t, ch), base + (size_t)min(t, n - 1) * ld + (size_t)(H + h) * DK + ch * 8);
    }
#pragma unroll
    for (int i = 0; i < 3 * DK * (NB / 8) / 128; i++) {
        const int e = tid + i * 128, d = e / (NB / 8), ch = e % (NB / 8);        // d: piece * DK + row of the state
        cp_async16(at(ss, VP, d, ch), S + (size_t)d * DV + ch * 8);
    }
#pragma unroll
    for (int i = 0; i < DC * (NB / 8) / 128; i++) {
        const int e = tid + i * 128, t = e / (NB / 8), ch = e % (NB / 8);
        cp_async16(at(vs, VP, t, ch), base + (size_t)min(t, n - 1) * ld + (size_t)2 * H * DK + (size_t)h * DV + col0 + ch * 8);
    }
    cp_async_commit();
    const int m0 = warp * 16, mi = lane >> 3, r = lane & 7;
    uint32_t qf[DK / 16][4];
    {
        const int row_a = min(m0 + (lane >> 2), n - 1), row_b = min(m0 + (lane >> 2) + 8, n - 1);
        const bf16 *qa = base + (size_t)row_a * ld + (size_t)h * DK + 2 * (lane & 3), *qb = base + (size_t)row_b * ld + (size_t)h * DK + 2 * (lane & 3);
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk++) {
            qf[kk][0] = *(const uint32_t *)(qa + kk * 16);
            qf[kk][1] = *(const uint32_t *)(qb + kk * 16);
            qf[kk][2] = *(const uint32_t *)(qa + kk * 16 + 8);
            qf[kk][3] = *(const uint32_t *)(qb + kk * 16 + 8);
        }
    }
    const float l2 = log2f(decay[h]);
    cp_async_wait<0>();
    __syncthreads();
    if (m0 >= n) return;
    float o[NB / 8][4], s[DC / 8][4];
#pragma unroll
    for (int d = 0; d < NB / 8; d++) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
#pragma unroll
    for (int j = 0; j < DC / 8; j++) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DK / 16; kk++) {
        const uint32_t (&a)[4] = qf[kk];
        // scores with the chunk's keys (those behind the warp's last token are masked below)
#pragma unroll
        for (int jj = 0; jj < DC / 16; jj++) {
            if (jj > warp) break;
            const int row = jj * 16 + (mi >> 1) * 8 + r, ch = kk * 2 + (mi & 1);
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(ks + row * KP + ((ch ^ (row & 7)) << 4), b0, b1, b2, b3);
            mma_bf16(s[2 * jj], a, b0, b1);
            mma_bf16(s[2 * jj + 1], a, b2, b3);
        }
        // what the state in front of the chunk gives
#pragma unroll
        for (int p = 2; p >= 0; p--)
#pragma unroll
            for (int dd = 0; dd < NB / 16; dd++) {
                const int row = kk * 16 + (mi & 1) * 8 + r, ch = dd * 2 + (mi >> 1);
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(ss + p * SPIECE + row * VP + ((ch ^ (row & 7)) << 4), b0, b1, b2, b3);
                mma_bf16(o[2 * dd], a, b0, b1);
                mma_bf16(o[2 * dd + 1], a, b2, b3);
            }
    }
    const int i0 = m0 + (lane >> 2), i1 = i0 + 8;
    const float f0 = exp2f(l2 * (float)(i0 + 1)), f1 = exp2f(l2 * (float)(i1 + 1));
#pragma unroll
    for (int d = 0; d < NB / 8; d++) { o[d][0] *= f0; o[d][1] *= f0; o[d][2] *= f1; o[d][3] *= f1; }
    // the chunk's own tokens: weights decay^(i-j) for j <= i
#pragma unroll
    for (int j = 0; j < DC / 8; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = e < 2 ? i0 : i1, t = j * 8 + 2 * (lane & 3) + (e & 1);
            s[j][e] = t <= i ? s[j][e] * exp2f(l2 * (float)(i - t)) : 0.f;
        }
#pragma unroll
    for (int kk = 0; kk < DC / 16; kk++) {
        if (kk > warp) break;
        uint32_t a[3][4];
        split3_pair(s[2 * kk][0], s[2 * kk][1], a[0][0], a[1][0], a[2][0]);
        split3_pair(s[2 * kk][2], s[2 * kk][3], a[0][1], a[1][1], a[2][1]);
        split3_pair(s[2 * kk + 1][0], s[2 * kk + 1][1], a[0][2], a[1][2], a[2][2]);
        split3_pair(s[2 * kk + 1][2], s[2 * kk + 1][3], a[0][3], a[1][3], a[2][3]);
#pragma unroll
        for (int dd = 0; dd < NB / 16; dd++) {
            const int row = kk * 16 + (mi & 1) * 8 + r, ch = dd * 2 + (mi >> 1);
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(vs + row * VP + ((ch ^ (row & 7)) << 4), b0, b1, b2, b3);
#pragma unroll
            for (int p = 2; p >= 0; p--) {
                mma_bf16(o[2 * dd], a[p], b0, b1);
                mma_bf16(o[2 * dd + 1], a[p], b2, b3);
            }
        }
    }
    float *dst = out + (size_t)(r0 + i0) * ldo + (size_t)h * DV + col0 + 2 * (lane & 3);
#pragma unroll
    for (int d = 0; d < NB / 8; d++) {
        if (i0 < n) *(float2 *)(dst + d * 8) = make_float2(o[d][0], o[d][1]);
        if (i1 < n) *(float2 *)(dst + (size_t)8 * ldo + d * 8) = make_float2(o[d][2], o[d][3]);
    }
}

// Single tokens and short portions: a block per (sequence, head) walks its tokens with the state in registers - thread (g, j) owns
// columns 4 j .. 4 j + 3 of rows g, g + RG, ...  The state rows are written by this entry's kernels alone, once a step, and slots by the
// copy that opens a step (see common.cuh), so the state is fetched before the wait on the projection.
template <int DK, int DV>
__global__ void __launch_bounds__(DA_THREADS)
decay_step_kernel(const bf16 *__restrict__ proj, int ld, float *__restrict__ out, int ldo, const int *__restrict__ cu_rows,
                  const int *__restrict__ slots, const float *__restrict__ decay, float *__restrict__ state, int H) {
    constexpr int NJ = DV / 4, RG = DA_THREADS / NJ, RPT = DK / RG;
    __shared__ float qs[DK], ks[DK];
    __shared__ __align__(16) float vs[DV], part[RG * DV];
    pdl_launch_dependents_small_step(gridDim.x);
    const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, j = tid % NJ, g = tid / NJ;
    const int row0 = cu_rows[seq], row1 = cu_rows[seq + 1];
    float4 *Sg = (float4 *)(state + ((size_t)slots[seq] * H + h) * DK * DV) + j;
    const float dec = decay[h];
    float4 S[RPT];
#pragma unroll
    for (int u = 0; u < RPT; u++) S[u] = Sg[(g + RG * u) * NJ];
    pdl_wait();
    if (row1 <= row0) return;
    for (int r = row0; r < row1; r++) {
        const bf16 *row = proj + (size_t)r * ld;
        for (int e = tid; e < 2 * DK + DV; e += DA_THREADS) {
            if (e < DK) qs[e] = da_act(row[(size_t)h * DK + e]);
            else if (e < 2 * DK) ks[e - DK] = da_act(row[(size_t)(H + h) * DK + e - DK]);
            else vs[e - 2 * DK] = da_act(row[(size_t)2 * H * DK + (size_t)h * DV + e - 2 * DK]);
        }
        __syncthreads();
        const float4 v = *(const float4 *)(vs + 4 * j);
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < RPT; u++) {
            const float k = ks[g + RG * u], q = qs[g + RG * u];
            S[u].x = fmaf(S[u].x, dec, k * v.x); S[u].y = fmaf(S[u].y, dec, k * v.y);
            S[u].z = fmaf(S[u].z, dec, k * v.z); S[u].w = fmaf(S[u].w, dec, k * v.w);
            acc.x = fmaf(S[u].x, q, acc.x); acc.y = fmaf(S[u].y, q, acc.y); acc.z = fmaf(S[u].z, q, acc.z); acc.w = fmaf(S[u].w, q, acc.w);
        }
        *(float4 *)(part + g * DV + 4 * j) = acc;
        __syncthreads();
        if (tid < DV) {
            float o = 0.f;
#pragma unroll
            for (int i = 0; i < RG; i++) o += part[i * DV + tid];
            out[(size_t)r * ldo + (size_t)h * DV + tid] = o;
        }
    }
#pragma unroll
    for (int u = 0; u < RPT; u++) Sg[(g + RG * u) * NJ] = S[u];
}

// out[m, :] = o[m, :] / sqrt(mean(o^2) + eps) * w * gate(g[m, :]), gate: sigmoid or silu; o float32, g and out bfloat16.  A block a row
// whose numbers stay in registers between the sum of squares and the output (C a multiple of 4, at most 4 RN threads).
template <int RN>
__global__ void __launch_bounds__(DA_THREADS)
row_norm_gate_kernel(const float *__restrict__ o, int ldo, const bf16 *__restrict__ g, int ldg, const float *__restrict__ w, bf16 *__restrict__ out,
                     int ldout, int C, float eps, int sigmoid_gate) {
    __shared__ float scratch[32];
    pdl_launch_dependents_small_step(gridDim.x);
    pdl_wait();
    const int m = blockIdx.x, tid = threadIdx.x;
    const float *src = o + (size_t)m * ldo;
    float4 v[RN];
    uint2 gr[RN];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < RN; i++) {
        const int c = (tid + i * DA_THREADS) * 4;
        v[i] = c < C ? *(const float4 *)(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        gr[i] = c < C ? *(const uint2 *)(g + (size_t)m * ldg + c) : make_uint2(0, 0);
    }
#pragma unroll
    for (int i = 0; i < RN; i++) { ss += v[i].x * v[i].x; ss += v[i].y * v[i].y; ss += v[i].z * v[i].z; ss += v[i].w * v[i].w; }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)C + eps);
#pragma unroll
    for (int i = 0; i < RN; i++) {
        const int c = (tid + i * DA_THREADS) * 4;
        if (c >= C) break;
        const float4 wc = *(const float4 *)(w + c);
        const bf16 *z = (const bf16 *)&gr[i];
        float t[4] = {v[i].x * inv * wc.x, v[i].y * inv * wc.y, v[i].z * inv * wc.z, v[i].w * inv * wc.w};
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const float zz = __bfloat162float(z[e]);
            t[e] *= (sigmoid_gate ? 1.0f : zz) / (1.0f + expf(-zz));
        }
        *(uint2 *)(out + (size_t)m * ldout + c) = make_uint2(pack_bf16(t[0], t[1]), pack_bf16(t[2], t[3]));
    }
}

// ------------------------------------------------------------------ launchers
extern "C" int fg_retention_plan(const int *cu_rows, int n_seq, int n_chunks, int chunk, int *plan, cudaStream_t stream);

extern "C" int fg_decay_attention_chunk_tokens(void) { return DC; }
extern "C" int fg_decay_attention_ok(int dk, int dv) { return (dk == 64 || dk == 128) && (dv == 64 || dv == 128); }

template <int DK, int DV>
static int decay_chunked(bf16 *proj, int ld, float *out, int ldo, const int *cu_rows, const int *slots, const float *decay, float *state, int *plan,
                         float *U, bf16 *P, int n_seq, int n_chunks, int H, cudaStream_t stream) {
    constexpr int smem_state = (3 * DC * DK + DC * DV) * 2, smem_out = (DC * DK + DC * 64 + 3 * DK * 64) * 2;
    static FgPerDevice setup;
    if (fg_needs_setup(setup)) {
        cudaError_t e = cudaFuncSetAttribute(decay_state_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_state);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_out);
        if (e != cudaSuccess) return (int)e;
    }
    const int *chunk_row = plan, *chunk_len = plan + n_chunks;
    int code = fg_retention_plan(cu_rows, n_seq, n_chunks, DC, plan, stream);
    if (code) return code;
    code = fg_launch(decay_state_kernel<DK, DV>, dim3(n_chunks, H), dim3(DA_THREADS), (size_t)smem_state, stream, proj, ld, chunk_row, chunk_len, decay, U, H);
    if (code) return code;
    code = fg_launch(decay_scan_kernel, dim3(n_seq, H, DK * DV / 4 / DA_THREADS), dim3(DA_THREADS), 0, stream, plan + 2 * n_chunks, chunk_len, slots, decay,
                     (const float *)U, P, state, H, DK * DV);
    if (code) return code;
    return fg_launch(decay_out_kernel<DK, DV>, dim3(n_chunks, H, DV / 64), dim3(128), (size_t)smem_out, stream, (const bf16 *)proj, ld, out, ldo, chunk_row, chunk_len, decay,
                     (const bf16 *)P, H);
}

static bool da_args_ok(const void *proj, int ld, const void *out, int ldo, const void *state, int H) {
    return H > 0 && H <= 65535 && ld % 8 == 0 && ldo % 4 == 0 && ((((uintptr_t)proj) | ((uintptr_t)out) | ((uintptr_t)state)) & 15) == 0;
}
#define DA_BY_SIZE(CALL) do { \
        if (dk == 64 && dv == 64) CALL(64, 64); \
        if (dk == 64 && dv == 128) CALL(64, 128); \
        if (dk == 128 && dv == 64) CALL(128, 64); \
        if (dk == 128 && dv == 128) CALL(128, 128); } while (0)

// proj [M, ld] bfloat16 rows q | k | v | g; state [slots, H, dk, dv] float32; out [M, H * dv] float32: the sums o.  n_chunks = sum over
// sequences of ceil(rows / fg_decay_attention_chunk_tokens()); plan: scratch of 2 * n_chunks + n_seq + 1 ints; U: scratch
// [n_chunks, H, dk, dv] float32; P: scratch [n_chunks, H, 3, dk, dv] bfloat16.  q, k and v of `proj` become their activations.  Decays
// must be positive.
extern "C" int fg_decay_attention_chunked(void *proj, int ld, float *out, int ldo, const int *cu_rows, const int *slots, const float *decay,
                                          float *state, int *plan, float *U, void *P, int n_seq, int n_chunks, int H, int dk, int dv,
                                          cudaStream_t stream) {
    if (n_seq <= 0 || n_chunks <= 0) return 0;
    if (!da_args_ok(proj, ld, out, ldo, state, H) || (((uintptr_t)U | (uintptr_t)P) & 15)) return FG_ERR_BAD_SIZE;
#define DA_CHUNKED(DK, DV) return decay_chunked<DK, DV>((bf16 *)proj, ld, out, ldo, cu_rows, slots, decay, state, plan, U, (bf16 *)P, n_seq, n_chunks, H, stream)
    DA_BY_SIZE(DA_CHUNKED);
#undef DA_CHUNKED
    return FG_ERR_BAD_SIZE;
}

extern "C" int fg_decay_attention_step(const void *proj, int ld, float *out, int ldo, const int *cu_rows, const int *slots, const float *decay,
                                       float *state, int n_seq, int H, int dk, int dv, cudaStream_t stream) {
    if (n_seq <= 0) return 0;
    if (!da_args_ok(proj, ld, out, ldo, state, H)) return FG_ERR_BAD_SIZE;
#define DA_STEP(DK, DV) return fg_launch(decay_step_kernel<DK, DV>, dim3(n_seq, H), dim3(DA_THREADS), 0, stream, (const bf16 *)proj, ld, out, ldo, cu_rows, slots, \
                                         decay, state, H)
    DA_BY_SIZE(DA_STEP);
#undef DA_STEP
    return FG_ERR_BAD_SIZE;
}

extern "C" int fg_row_norm_gate(const float *o, int ldo, const void *g, int ldg, const float *w, void *out, int ldout, int M, int C, float eps,
                                int sigmoid_gate, cudaStream_t stream) {
    if (M <= 0) return 0;
    if (C <= 0 || C % 4 || C > 4 * DA_THREADS * 8 || ldo % 4 || ldg % 4 || ldout % 4 || ((((uintptr_t)o) | ((uintptr_t)w)) & 15) ||
        ((((uintptr_t)g) | ((uintptr_t)out)) & 7))
        return FG_ERR_BAD_SIZE;
    const int rn = (C + 4 * DA_THREADS - 1) / (4 * DA_THREADS);
#define RNG_RUN(RN) return fg_launch(row_norm_gate_kernel<RN>, dim3(M), dim3(DA_THREADS), 0, stream, o, ldo, (const bf16 *)g, ldg, w, (bf16 *)out, ldout, C, eps, \
                                     sigmoid_gate)
    if (rn == 1) RNG_RUN(1);
    if (rn == 2) RNG_RUN(2);
    if (rn <= 4) RNG_RUN(4);
    RNG_RUN(8);
#undef RNG_RUN
}
