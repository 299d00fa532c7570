// mlstm.cuh -- device kernels of the matrix memory with exponential gates (mLSTM) of layered plans.  First user: Kegasun.
//
// Per head, over the rows of a launch, with i, f the log gates of the row and S [dk][dv], n [dk], m carried from launch to launch:
//     m' = max(f + m, i);   a = exp(f + m - m');   b = exp(i - m');
//     S <- a S + b k v^T;   n <- a n + b k;   out = S^T q,   den = max(|<n, q>|, exp(-m')) + 1e-6
//   * k_mlstm_scan<R>  the state in registers: sixteen lanes share a column of S, lane `slice` holds R of its rows (the layout of
//                      k_ssd_scan); n is one more column whose value is 1, kept by a ninth warp of the head's first CTA;
//   * k_mlstm_scan_any the same for key sizes above 512: the state stays in global memory.
// The gates are evaluated here from the projection's logits (soft cap, log sigmoid); the running maximum of a batch of tokens is a
// max-plus scan over the lanes.  Everything is FP32 in both compute modes.  The read-out is finished by k_head_norm_gate.
#pragma once
#include "delta.cuh"
#include "recurrent.cuh"

namespace ly {

struct MlstmArgs {
    int heads, dk, dv;
    int q_off, k_off, v_off, i_off, f_off; // columns of a projection row
    const float *i_bias, *f_bias;          // [heads]
    float cap, q_scale;
    int vec;                               // 1: dk, the column offsets and the row stride are multiples of 4 floats
};
#define MLSTM_COLS 16
#define MLSTM_THREADS (MLSTM_COLS * 16 + 32)           // eight warps of columns, one for the normaliser (and for staging)
#define MLSTM_TB_OF(R) ((R) >= 32 ? 4 : (R) >= 16 ? 8 : 16) // tokens per staged batch: two buffers of k and q rows in 32 KB
__host__ __device__ inline int mlstm_reg_rows(int dk) { const int q = (dk + 15) / 16; return q <= 1 ? 1 : q <= 2 ? 2 : q <= 4 ? 4 : q <= 8 ? 8 : q <= 16 ? 16 : q <= 32 ? 32 : 0; }
__host__ __device__ inline int mlstm_tiles(int dk, int dv) { return mlstm_reg_rows(dk) ? (dv + MLSTM_COLS - 1) / MLSTM_COLS : (dv + 1 + 31) / 32; }
// State of one layer run: [head][tile][row of a lane][lane of the tile] columns, then [head][R][16] normalisers, then [head][tile] running maxima
// (a copy per CTA: no CTA reads what another one of the same launch writes).
__host__ __device__ inline size_t mlstm_state_floats(int heads, int dk, int dv) {
    const int R = mlstm_reg_rows(dk), tiles = mlstm_tiles(dk, dv);
    return R ? (size_t)heads * ((size_t)tiles * R * MLSTM_COLS * 16 + (size_t)R * 16 + tiles) : (size_t)heads * ((size_t)dk * (dv + 1) + tiles);
}

__device__ __forceinline__ float softcapf_(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float logsigmoidf_(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// grid (heads, tiles), MLSTM_THREADS threads.  Y row: [out: heads * dv | den: heads].
template <int R>
__global__ void __launch_bounds__(MLSTM_THREADS) k_mlstm_scan(const float *__restrict__ P, int ldp, MlstmArgs a, float *__restrict__ S, int n, const StepState *__restrict__ st,
                                                              float *__restrict__ Y, int ldy) {
    constexpr int RW = R * 16, TB = MLSTM_TB_OF(R);
    __shared__ __align__(16) float ks[2][TB][RW], qs[2][TB][RW];
    __shared__ float vs[2][TB][MLSTM_COLS], gs[2][2][16];
    const int h = blockIdx.x, tile = blockIdx.y, tiles = gridDim.y, tid = threadIdx.x, slice = tid & 15, cc = tid >> 4, col = tile * MLSTM_COLS + cc;
    const bool column = cc < MLSTM_COLS && col < a.dv, norm = tile == 0 && cc == MLSTM_COLS; // what this group of sixteen lanes keeps
    float *Sc = S + ((size_t)h * tiles + tile) * R * (MLSTM_COLS * 16) + tid;
    float *Sn = S + (size_t)a.heads * tiles * R * (MLSTM_COLS * 16) + (size_t)h * R * 16 + slice;
    float *Sm = S + (size_t)a.heads * ((size_t)tiles * R * (MLSTM_COLS * 16) + (size_t)R * 16) + (size_t)h * tiles + tile;
    const int ko = a.k_off + h * a.dk, qo = a.q_off + h * a.dk, vo = a.v_off + h * a.dv + tile * MLSTM_COLS;
    // rows beyond dk and tokens beyond n are zero
    auto fetch = [&](int t0, int buf) {
        const int nt = n - t0 < TB ? n - t0 : TB;
        if (a.vec) {
            for (int e = tid; e < TB * (RW / 4); e += MLSTM_THREADS) {
                const int t = e / (RW / 4), i = (e % (RW / 4)) * 4;
                const bool ok = t < nt && i < a.dk;
                const float *row = P + (size_t)(t0 + (ok ? t : 0)) * ldp;
                cp_async16(&ks[buf][t][i], ok ? row + ko + i : P, ok);
                cp_async16(&qs[buf][t][i], ok ? row + qo + i : P, ok);
            }
        } else {
            for (int e = tid; e < TB * RW; e += MLSTM_THREADS) {
                const int t = e / RW, i = e % RW;
                const bool ok = t < nt && i < a.dk;
                const float *row = P + (size_t)(t0 + (ok ? t : 0)) * ldp;
                cp_async4(&ks[buf][t][i], ok ? row + ko + i : P, ok);
                cp_async4(&qs[buf][t][i], ok ? row + qo + i : P, ok);
            }
        }
        for (int e = tid; e < TB * MLSTM_COLS; e += MLSTM_THREADS) {
            const int t = e / MLSTM_COLS, i = e % MLSTM_COLS;
            const bool ok = t < nt && tile * MLSTM_COLS + i < a.dv;
            cp_async4(&vs[buf][t][i], ok ? P + (size_t)(t0 + t) * ldp + vo + i : P, ok);
        }
        if (tid < 32) {
            const int t = tid & 15;
            const bool ok = t < nt;
            cp_async4(&gs[buf][tid >> 4][t], ok ? P + (size_t)(t0 + t) * ldp + (tid < 16 ? a.i_off : a.f_off) + h : P, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    const bool fresh = st->pos == 0;
    float s[R];
#pragma unroll
    for (int i = 0; i < R; i++) s[i] = fresh ? 0.0f : column ? Sc[(size_t)i * (MLSTM_COLS * 16)] : norm ? Sn[i * 16] : 0.0f;
    float m0 = fresh ? 0.0f : *Sm;
    const float ib = a.i_bias[h], fb = a.f_bias[h];
    int buf = 0;
    for (int t0 = 0; t0 < n; t0 += TB, buf ^= 1) {
        const int nt = n - t0 < TB ? n - t0 : TB;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads(); // this batch has landed for every thread, and the other buffer's batch is consumed
        if (t0 + TB < n) fetch(t0 + TB, buf ^ 1);
        // token `slice` of the batch: log gates, running maximum (max-plus scan over the lanes), decay, write strength, floor of the denominator
        const float il = softcapf_(gs[buf][0][slice] + ib, a.cap), fl = logsigmoidf_(softcapf_(gs[buf][1][slice] + fb, a.cap));
        float F = fl, M = il;
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) {
            const float Fp = __shfl_up_sync(0xffffffffu, F, o, 16), Mp = __shfl_up_sync(0xffffffffu, M, o, 16);
            if (slice >= o) { M = fmaxf(Mp + F, M); F += Fp; }
        }
        const float mt = fmaxf(m0 + F, M);
        float mp = __shfl_up_sync(0xffffffffu, mt, 1, 16);
        if (slice == 0) mp = m0;
        const float my_dec = expf(fl + mp - mt), my_wr = expf(il - mt), my_floor = expf(-mt);
        m0 = __shfl_sync(0xffffffffu, mt, nt - 1, 16);
        int tb = 0;
        for (; tb + 4 <= nt; tb += 4) { // four tokens: four independent read-out sums, reduced over the sixteen lanes with five shuffles
            float acc[4];
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const int t = tb + u;
                const float dA = __shfl_sync(0xffffffffu, my_dec, t, 16), wr = __shfl_sync(0xffffffffu, my_wr, t, 16);
                const float dx = wr * (cc < MLSTM_COLS ? vs[buf][t][cc] : 1.0f);
                float kv[R], qv[R];
                ssd_rows<R>(ks[buf][t], slice, kv);
                ssd_rows<R>(qs[buf][t], slice, qv);
                float ac = 0.0f;
#pragma unroll
                for (int i = 0; i < R; i++) {
                    s[i] = fmaf(dA, s[i], dx * kv[i]);
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
            const float floor_t = __shfl_sync(0xffffffffu, my_floor, t, 16);
            v *= a.q_scale;
            if ((slice & 3) == 0) {
                if (column) Y[(size_t)(t0 + t) * ldy + (size_t)h * a.dv + col] = v;
                else if (norm) Y[(size_t)(t0 + t) * ldy + (size_t)a.heads * a.dv + h] = fmaxf(fabsf(v), floor_t) + 1e-6f;
            }
        }
        for (int t = tb; t < nt; t++) {
            const float dA = __shfl_sync(0xffffffffu, my_dec, t, 16), wr = __shfl_sync(0xffffffffu, my_wr, t, 16), floor_t = __shfl_sync(0xffffffffu, my_floor, t, 16);
            const float dx = wr * (cc < MLSTM_COLS ? vs[buf][t][cc] : 1.0f);
            float kv[R], qv[R];
            ssd_rows<R>(ks[buf][t], slice, kv);
            ssd_rows<R>(qs[buf][t], slice, qv);
            float acc = 0.0f;
#pragma unroll
            for (int i = 0; i < R; i++) {
                s[i] = fmaf(dA, s[i], dx * kv[i]);
                acc = fmaf(s[i], qv[i], acc);
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 8);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc *= a.q_scale;
            if (slice == 0) {
                if (column) Y[(size_t)(t0 + t) * ldy + (size_t)h * a.dv + col] = acc;
                else if (norm) Y[(size_t)(t0 + t) * ldy + (size_t)a.heads * a.dv + h] = fmaxf(fabsf(acc), floor_t) + 1e-6f;
            }
        }
    }
#pragma unroll
    for (int i = 0; i < R; i++) {
        if (column) Sc[(size_t)i * (MLSTM_COLS * 16)] = s[i];
        else if (norm) Sn[i * 16] = s[i];
    }
    if (tid == 0) *Sm = m0;
}

// Any key size: grid (heads, ceil((dv + 1) / 32)), 256 threads = 32 columns x 8 row slices; column dv is the normaliser (value 1).  State: [head]
// [dk][dv + 1], then [head][tile] running maxima.
__global__ void __launch_bounds__(256) k_mlstm_scan_any(const float *__restrict__ P, int ldp, MlstmArgs a, float *__restrict__ S, int n, const StepState *__restrict__ st,
                                                        float *__restrict__ Y, int ldy) {
    __shared__ float part[8][33];
    const int h = blockIdx.x, tid = threadIdx.x, c = tid & 31, sl = tid >> 5, W = a.dv + 1, col = blockIdx.y * 32 + c;
    const bool live = col < W;
    float *Sg = S + (size_t)h * a.dk * W + col, *Sm = S + (size_t)a.heads * a.dk * W + (size_t)h * gridDim.y + blockIdx.y;
    const bool fresh = st->pos == 0;
    float m = fresh ? 0.0f : *Sm;
    for (int t = 0; t < n; t++) {
        const float *p = P + (size_t)t * ldp;
        const float il = softcapf_(p[a.i_off + h] + a.i_bias[h], a.cap), fl = logsigmoidf_(softcapf_(p[a.f_off + h] + a.f_bias[h], a.cap));
        const float m1 = fmaxf(fl + m, il), dA = expf(fl + m - m1), wr = expf(il - m1);
        m = m1;
        const float x = !live ? 0.0f : col < a.dv ? p[a.v_off + (size_t)h * a.dv + col] : 1.0f, dx = wr * x;
        const float *k = p + a.k_off + (size_t)h * a.dk, *q = p + a.q_off + (size_t)h * a.dk;
        float acc = 0.0f;
        if (live)
            for (int i = sl; i < a.dk; i += 8) {
                float s = (fresh && t == 0) ? 0.0f : Sg[(size_t)i * W];
                s = fmaf(dA, s, dx * k[i]);
                Sg[(size_t)i * W] = s;
                acc = fmaf(s, q[i], acc);
            }
        part[sl][c] = acc;
        __syncthreads();
        if (sl == 0 && live) {
            float v = 0.0f;
#pragma unroll
            for (int j = 0; j < 8; j++) v += part[j][c];
            v *= a.q_scale;
            if (col < a.dv) Y[(size_t)t * ldy + (size_t)h * a.dv + col] = v;
            else Y[(size_t)t * ldy + (size_t)a.heads * a.dv + h] = fmaxf(fabsf(v), expf(-m)) + 1e-6f;
        }
        __syncthreads();
    }
    if (tid == 0) *Sm = m;
}

} // namespace ly
