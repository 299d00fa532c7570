// lightning.cuh -- device kernels of the decayed linear attention of layered plans (B200_MIXER_LIGHTNING).  First user: Zulesun.
//
// Per head, over the rows of a launch, S [dk][dv] carried from launch to launch (zero at position 0), c a constant of the head:
//     q = silu(q'), k = silu(k'), v = silu(v');   S <- c S + k v^T;   o = S^T q
//   * k_lightning_scan<R>  token by token in FP32, the state in registers: sixteen lanes share a column of S, lane `slice` holds R of its rows
//                          (ssd_rows); projections staged through shared memory with the activation applied on the way;
//   * k_lightning_chunk<DK>  the same for a prefill chunk of BF16 plans, on the tensor cores (mma.sync m16n8k16): q, k, v rounded to BF16 behind their
//                          activation (what a BF16 plan may do), 64 tokens at a time
//                              o_t = sum_{s <= t} c^(t-s) <q_t, k_s> v_s + c^(t+1) S^T q_t,   S <- c^64 S + sum_s c^(63-s) k_s v_s^T.
//                          Everything behind the activations stays 32-bit: scores and decays are FP32, S accumulates in FP32 registers, and every FP32
//                          operand of a product (decayed score, decayed value, S) enters as the sum of two BF16 numbers (its rounding and the
//                          rounding of the rest, 16 bits together) against an exact BF16 operand.
// The state is kept as its transpose, [head][dv][lightning_rows(dk)] floats: a column is contiguous (rows beyond dk stay zero).
// The read-out is finished by k_gated_group_norm.
#pragma once
#include "recurrent.cuh"

namespace ly {

struct LightningArgs {
    int heads, dk, dv;
    int q_off, k_off, v_off; // columns of a projection row
    const float *decay;      // [heads]
};
#define LIGHT_COLS 16
#define LIGHT_THREADS (LIGHT_COLS * 16)
__host__ __device__ inline int lightning_reg_rows(int dk) { const int q = (dk + 15) / 16; return q <= 1 ? 1 : q <= 2 ? 2 : q <= 4 ? 4 : q <= 8 ? 8 : q <= 16 ? 16 : q <= 32 ? 32 : 0; }
__host__ __device__ inline int lightning_rows(int dk) { return 16 * lightning_reg_rows(dk); }
__host__ __device__ inline size_t lightning_state_floats(int heads, int dk, int dv) { return (size_t)heads * dv * lightning_rows(dk); }

__device__ __forceinline__ float siluf_(float z) { return z / (1.0f + expf(-z)); }

// grid (heads, ceil(dv / LIGHT_COLS)), LIGHT_THREADS threads.  Y [n][ldy]: read-outs [heads][dv].
template <int R>
__global__ void __launch_bounds__(LIGHT_THREADS) k_lightning_scan(const float *__restrict__ P, int ldp, LightningArgs a, float *__restrict__ S, int n, const StepState *__restrict__ st,
                                                                  float *__restrict__ Y, int ldy) {
    constexpr int RW = R * 16, TB = R >= 32 ? 4 : R >= 16 ? 8 : 16, LB = TB * RW / LIGHT_THREADS;
    __shared__ __align__(16) float ks[2][TB][RW], qs[2][TB][RW];
    __shared__ float vs[2][TB][LIGHT_COLS];
    const int h = blockIdx.x, tid = threadIdx.x, slice = tid & 15, cc = tid >> 4, j0 = blockIdx.y * LIGHT_COLS, col = j0 + cc;
    const bool column = col < a.dv;
    const int qo = a.q_off + h * a.dk, ko = a.k_off + h * a.dk, vo = a.v_off + h * a.dv + j0;
    float pk[LB], pq[LB], pv = 0.0f; // the next batch on its way to shared memory
    auto load = [&](int t0) {
        const int nt = n - t0 < TB ? n - t0 : TB;
#pragma unroll
        for (int k = 0; k < LB; k++) {
            const int e = tid + k * LIGHT_THREADS, t = e / RW, i = e % RW;
            const bool ok = t < nt && i < a.dk;
            const float *row = P + (size_t)(ok ? t0 + t : 0) * ldp;
            pk[k] = ok ? row[ko + i] : 0.0f;
            pq[k] = ok ? row[qo + i] : 0.0f;
        }
        if (tid < TB * LIGHT_COLS) {
            const int t = tid / LIGHT_COLS, i = tid % LIGHT_COLS;
            pv = t < nt && j0 + i < a.dv ? P[(size_t)(t0 + t) * ldp + vo + i] : 0.0f;
        }
    };
    auto store = [&](int buf, int nt) { // silu(0) = 0: rows beyond dk stay zero; nothing reads a token beyond the end
#pragma unroll
        for (int k = 0; k < LB; k++) {
            const int e = tid + k * LIGHT_THREADS;
            if (e / RW >= nt) continue;
            (&ks[buf][0][0])[e] = siluf_(pk[k]);
            (&qs[buf][0][0])[e] = siluf_(pq[k]);
        }
        if (tid < TB * LIGHT_COLS && tid / LIGHT_COLS < nt) (&vs[buf][0][0])[tid] = siluf_(pv);
    };
    load(0);
    float *Sg = S + ((size_t)h * a.dv + (column ? col : 0)) * RW;
    float s[R];
    if (column && st->pos != 0) ssd_rows<R>(Sg, slice, s);
    else {
#pragma unroll
        for (int i = 0; i < R; i++) s[i] = 0.0f;
    }
    const float dec = a.decay[h];
    store(0, n < TB ? n : TB);
    __syncthreads();
    int buf = 0;
    for (int t0 = 0; t0 < n; t0 += TB, buf ^= 1) {
        const int nt = n - t0 < TB ? n - t0 : TB;
        const bool more = t0 + TB < n;
        if (more) load(t0 + TB);
        int tb = 0;
        for (; tb + 4 <= nt; tb += 4) { // four tokens: four independent read-out sums, reduced over the sixteen lanes with five shuffles
            float acc[4];
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const float x = vs[buf][tb + u][cc];
                float kv[R], qv[R];
                ssd_rows<R>(ks[buf][tb + u], slice, kv);
                ssd_rows<R>(qs[buf][tb + u], slice, qv);
                float ac = 0.0f;
#pragma unroll
                for (int i = 0; i < R; i++) {
                    s[i] = fmaf(dec, s[i], x * kv[i]);
                    ac = fmaf(s[i], qv[i], ac);
                }
                acc[u] = ac;
            }
            const bool hi8 = slice & 8, hi4 = slice & 4;
            float p0 = hi8 ? acc[2] : acc[0], p1 = hi8 ? acc[3] : acc[1];
            p0 += __shfl_xor_sync(0xffffffffu, hi8 ? acc[0] : acc[2], 8);
            p1 += __shfl_xor_sync(0xffffffffu, hi8 ? acc[1] : acc[3], 8);
            float v = hi4 ? p1 : p0;
            v += __shfl_xor_sync(0xffffffffu, hi4 ? p0 : p1, 4);
            v += __shfl_xor_sync(0xffffffffu, v, 2);
            v += __shfl_xor_sync(0xffffffffu, v, 1);
            const int t = tb + (slice >> 2); // lanes 0, 4, 8, 12 of a column hold the sums of tokens tb .. tb + 3
            if ((slice & 3) == 0 && column) Y[(size_t)(t0 + t) * ldy + (size_t)h * a.dv + col] = v;
        }
        for (int t = tb; t < nt; t++) {
            const float x = vs[buf][t][cc];
            float kv[R], qv[R];
            ssd_rows<R>(ks[buf][t], slice, kv);
            ssd_rows<R>(qs[buf][t], slice, qv);
            float acc = 0.0f;
#pragma unroll
            for (int i = 0; i < R; i++) {
                s[i] = fmaf(dec, s[i], x * kv[i]);
                acc = fmaf(s[i], qv[i], acc);
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 8);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            if (slice == 0 && column) Y[(size_t)(t0 + t) * ldy + (size_t)h * a.dv + col] = acc;
        }
        if (more) store(buf ^ 1, n - t0 - TB < TB ? n - t0 - TB : TB); // that buffer was consumed before the barrier that started this iteration
        __syncthreads();
    }
    if (!column) return;
    if constexpr (R % 4 == 0) {
#pragma unroll
        for (int k = 0; k < R / 4; k++) *reinterpret_cast<float4 *>(Sg + (16 * k + slice) * 4) = make_float4(s[4 * k], s[4 * k + 1], s[4 * k + 2], s[4 * k + 3]);
    } else {
#pragma unroll
        for (int i = 0; i < R; i++) Sg[slice * R + i] = s[i];
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// grid (heads, ceil(dv / COLS)), 4 * COLS threads (COLS = 64, or 32 where that fills more SMs), dynamic shared memory lightning_chunk_smem<DK, COLS>.  QKV [n][ld]: [q: heads * DK | k: heads * DK |
// v: heads * dv] behind the activation; dv a multiple of 8, ld a multiple of 8.  A CTA walks the chunk's tokens LC_TOKENS at a time (next tile in flight by
// cp.async) for COLS columns of one head's state.  Warp w: read-out of token rows 16 (w & 3) .. for 32 of the columns; state columns (rows of the
// transpose) 16 (w mod COLS / 16) .. for half of the DK entries, as accumulator fragments of the update product.
// ---------------------------------------------------------------------------------------------------------------------
#define LC_TOKENS 64
template <int DK, int COLS> __host__ __device__ constexpr size_t lightning_chunk_smem() { // Q, K x 2 buffers, V x 2, split decayed V, split S^T
    return (size_t)2 * (4 * LC_TOKENS * (DK + 8) + 2 * LC_TOKENS * (COLS + 8) + 2 * LC_TOKENS * (COLS + 8) + 2 * COLS * (DK + 8));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void *row) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
// x, y -> packed BF16 roundings and packed roundings of what they leave
__device__ __forceinline__ void split_bf16(float x, float y, unsigned &hi, unsigned &lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - bf_lo(hi), y - bf_hi(hi));
}

template <int DK, int COLS>
__global__ void __launch_bounds__(4 * COLS) k_lightning_chunk(const bf16 *__restrict__ QKV, int ld, LightningArgs a, float *__restrict__ S, int n, const StepState *__restrict__ st,
                                                                float *__restrict__ Y, int ldy) {
    extern __shared__ __align__(16) unsigned char lsm[];
    constexpr int T = LC_TOKENS, QW = DK + 8, VW = COLS + 8, LC_THREADS = 4 * COLS, LC_COLS = COLS;
    typedef bf16 QRow[QW];
    typedef bf16 VRow[VW];
    QRow *Qs = reinterpret_cast<QRow *>(lsm), *Ks = Qs + 2 * T; // [buffer * T + token]
    QRow *SH = Ks + 2 * T, *SL = SH + LC_COLS;                 // [state column]
    VRow *Vs = reinterpret_cast<VRow *>(SL + LC_COLS), *VH = Vs + 2 * T, *VL = VH + T;
    __shared__ float pw[T + 1]; // powers of the head's decay
    const int h = blockIdx.x, j0 = blockIdx.y * LC_COLS, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int rb = (warp & 3) * 16, half = warp >> 2;                           // read-out: token rows, block of 32 columns
    const int sb = warp % (COLS / 16) * 16, shalf = warp / (COLS / 16);         // state: columns, half of the DK entries
    const int qo = h * DK, ko = a.heads * DK + h * DK, vo = 2 * a.heads * DK + h * a.dv + j0;
    auto fetch = [&](int t0, int buf) {
        const int nt = n - t0 < T ? n - t0 : T;
        for (int e = tid; e < T * (DK / 8); e += LC_THREADS) {
            const int r = e / (DK / 8), c = (e % (DK / 8)) * 8;
            const bool ok = r < nt;
            const bf16 *row = QKV + (size_t)(ok ? t0 + r : 0) * ld;
            cp_async16(&Qs[buf * T + r][c], row + qo + c, ok);
            cp_async16(&Ks[buf * T + r][c], row + ko + c, ok);
        }
        for (int e = tid; e < T * (LC_COLS / 8); e += LC_THREADS) {
            const int r = e / (LC_COLS / 8), c = (e % (LC_COLS / 8)) * 8;
            const bool ok = r < nt && j0 + c < a.dv;
            cp_async16(&Vs[buf * T + r][c], ok ? QKV + (size_t)(t0 + r) * ld + vo + c : QKV, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    for (int i = tid; i <= T; i += LC_THREADS) pw[i] = powf(a.decay[h], (float)i);
    // S^T rows j0 + sb + g (+ 8), entries shalf * DK / 2 + i * 8 + 2 t (+ 1)
    float s[DK / 16][4];
    float *Sg = S + ((size_t)h * a.dv + j0 + sb + g) * DK + shalf * (DK / 2) + 2 * t;
    const bool in0 = j0 + sb + g < a.dv, in1 = j0 + sb + g + 8 < a.dv, fresh = st->pos == 0;
#pragma unroll
    for (int i = 0; i < DK / 16; i++) {
        const float2 z = make_float2(0.0f, 0.0f);
        const float2 u = in0 && !fresh ? *reinterpret_cast<const float2 *>(Sg + i * 8) : z, v = in1 && !fresh ? *reinterpret_cast<const float2 *>(Sg + (size_t)8 * DK + i * 8) : z;
        s[i][0] = u.x; s[i][1] = u.y; s[i][2] = v.x; s[i][3] = v.y;
    }
    int buf = 0;
    for (int t0 = 0; t0 < n; t0 += T, buf ^= 1) {
        const int nt = n - t0 < T ? n - t0 : T;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads(); // this tile has landed for every thread; the other buffer and the split operands are free
        if (t0 + T < n) fetch(t0 + T, buf ^ 1);
        const QRow *Q = Qs + buf * T, *K = Ks + buf * T;
        const VRow *V = Vs + buf * T;
#pragma unroll
        for (int i = 0; i < DK / 16; i++) {
            unsigned hi, lo;
            const int c = shalf * (DK / 2) + i * 8 + 2 * t;
            split_bf16(s[i][0], s[i][1], hi, lo);
            *reinterpret_cast<unsigned *>(&SH[sb + g][c]) = hi; *reinterpret_cast<unsigned *>(&SL[sb + g][c]) = lo;
            split_bf16(s[i][2], s[i][3], hi, lo);
            *reinterpret_cast<unsigned *>(&SH[sb + g + 8][c]) = hi; *reinterpret_cast<unsigned *>(&SL[sb + g + 8][c]) = lo;
        }
        for (int e = tid; e < T * (LC_COLS / 2); e += LC_THREADS) {
            const int r = e / (LC_COLS / 2), c = (e % (LC_COLS / 2)) * 2;
            const unsigned v = *reinterpret_cast<const unsigned *>(&V[r][c]);
            const float f = r < nt ? pw[nt - 1 - r] : 0.0f;
            unsigned hi, lo;
            split_bf16(bf_lo(v) * f, bf_hi(v) * f, hi, lo);
            *reinterpret_cast<unsigned *>(&VH[r][c]) = hi; *reinterpret_cast<unsigned *>(&VL[r][c]) = lo;
        }
        __syncthreads();
        if (rb < nt) { // read-out of this warp's sixteen tokens
            unsigned qf[DK / 16][4];
#pragma unroll
            for (int kk = 0; kk < DK / 16; kk++) {
                qf[kk][0] = *reinterpret_cast<const unsigned *>(&Q[rb + g][kk * 16 + 2 * t]);
                qf[kk][1] = *reinterpret_cast<const unsigned *>(&Q[rb + g + 8][kk * 16 + 2 * t]);
                qf[kk][2] = *reinterpret_cast<const unsigned *>(&Q[rb + g][kk * 16 + 2 * t + 8]);
                qf[kk][3] = *reinterpret_cast<const unsigned *>(&Q[rb + g + 8][kk * 16 + 2 * t + 8]);
            }
            float o[4][4];
#pragma unroll
            for (int j = 0; j < 4; j++) {
#pragma unroll
                for (int e = 0; e < 4; e++) o[j][e] = 0.0f;
#pragma unroll
                for (int kk = 0; kk < DK / 16; kk++) { // what the state held before these tokens
                    const int r = half * 32 + j * 8 + g;
                    unsigned b[2];
                    b[0] = *reinterpret_cast<const unsigned *>(&SH[r][kk * 16 + 2 * t]); b[1] = *reinterpret_cast<const unsigned *>(&SH[r][kk * 16 + 2 * t + 8]);
                    mma_bf16_16816(o[j], qf[kk], b);
                    b[0] = *reinterpret_cast<const unsigned *>(&SL[r][kk * 16 + 2 * t]); b[1] = *reinterpret_cast<const unsigned *>(&SL[r][kk * 16 + 2 * t + 8]);
                    mma_bf16_16816(o[j], qf[kk], b);
                }
                const float d0 = pw[rb + g + 1], d1 = pw[rb + g + 9];
                o[j][0] *= d0; o[j][1] *= d0; o[j][2] *= d1; o[j][3] *= d1;
            }
#pragma unroll
            for (int kb = 0; kb < T / 16; kb++) { // sixteen keys at a time: scores, decay and mask, values
                if (kb * 16 > rb) break;          // later than every token of this warp
                float p[2][4];
#pragma unroll
                for (int u = 0; u < 2; u++) {
#pragma unroll
                    for (int e = 0; e < 4; e++) p[u][e] = 0.0f;
#pragma unroll
                    for (int kk = 0; kk < DK / 16; kk++) {
                        const int r = kb * 16 + u * 8 + g;
                        unsigned b[2];
                        b[0] = *reinterpret_cast<const unsigned *>(&K[r][kk * 16 + 2 * t]); b[1] = *reinterpret_cast<const unsigned *>(&K[r][kk * 16 + 2 * t + 8]);
                        mma_bf16_16816(p[u], qf[kk], b);
                    }
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int back = rb + g + (e >> 1) * 8 - (kb * 16 + u * 8 + 2 * t + (e & 1));
                        p[u][e] = back >= 0 ? p[u][e] * pw[back] : 0.0f;
                    }
                }
                unsigned ph[4], pl[4];
                split_bf16(p[0][0], p[0][1], ph[0], pl[0]); split_bf16(p[0][2], p[0][3], ph[1], pl[1]);
                split_bf16(p[1][0], p[1][1], ph[2], pl[2]); split_bf16(p[1][2], p[1][3], ph[3], pl[3]);
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    unsigned b[2];
                    ldmatrix_x2_trans(b, &V[kb * 16 + (lane & 15)][half * 32 + j * 8]);
                    mma_bf16_16816(o[j], ph, b);
                    mma_bf16_16816(o[j], pl, b);
                }
            }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int c = j0 + half * 32 + j * 8 + 2 * t; // dv is a multiple of 8: both entries or none
                if (c >= a.dv) continue;
                float *y = Y + (size_t)(t0 + rb + g) * ldy + (size_t)h * a.dv + c;
                if (rb + g < nt) *reinterpret_cast<float2 *>(y) = make_float2(o[j][0], o[j][1]);
                if (rb + g + 8 < nt) *reinterpret_cast<float2 *>(y + (size_t)8 * ldy) = make_float2(o[j][2], o[j][3]);
            }
        }
        // state: decayed, plus the products of this tile's keys and decayed values
        const float dn = pw[nt];
#pragma unroll
        for (int i = 0; i < DK / 16; i++) { s[i][0] *= dn; s[i][1] *= dn; s[i][2] *= dn; s[i][3] *= dn; }
#pragma unroll
        for (int kk = 0; kk < T / 16; kk++) {
            unsigned vh[4], vl[4];
            const int r = kk * 16 + (lane >> 4) * 8 + (lane & 7), c = sb + ((lane >> 3) & 1) * 8; // four 8 x 8 blocks, transposed: [value][token]
            ldmatrix_x4_trans(vh, &VH[r][c]);
            ldmatrix_x4_trans(vl, &VL[r][c]);
#pragma unroll
            for (int i = 0; i < DK / 16; i++) {
                unsigned b[2];
                ldmatrix_x2_trans(b, &K[kk * 16 + (lane & 15)][shalf * (DK / 2) + i * 8]);
                mma_bf16_16816(s[i], vh, b);
                mma_bf16_16816(s[i], vl, b);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < DK / 16; i++) {
        if (in0) *reinterpret_cast<float2 *>(Sg + i * 8) = make_float2(s[i][0], s[i][1]);
        if (in1) *reinterpret_cast<float2 *>(Sg + (size_t)8 * DK + i * 8) = make_float2(s[i][2], s[i][3]);
    }
}

} // namespace ly
