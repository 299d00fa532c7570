// lightning.cuh -- device kernels of the decayed linear attention of layered plans (B200_MIXER_LIGHTNING).  First user: Zulesun.
//
// Per head, over the rows of a launch, S [dk][dv] carried from launch to launch (zero at position 0), c a constant of the head:
//     q = silu(q'), k = silu(k'), v = silu(v');   S <- c S + k v^T;   o = S^T q
//   * k_lightning_scan<R>  token by token in FP32, the state in registers: sixteen lanes share a column of S, lane `slice` holds R of its rows
//                          (ssd_rows); projections staged through shared memory with the activation applied on the way.
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
    auto store = [&](int buf) { // silu(0) = 0: rows and tokens beyond the end stay zero
#pragma unroll
        for (int k = 0; k < LB; k++) {
            const int e = tid + k * LIGHT_THREADS;
            (&ks[buf][0][0])[e] = siluf_(pk[k]);
            (&qs[buf][0][0])[e] = siluf_(pq[k]);
        }
        if (tid < TB * LIGHT_COLS) (&vs[buf][0][0])[tid] = siluf_(pv);
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
    store(0);
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
        if (more) store(buf ^ 1); // that buffer was consumed before the barrier that started this iteration
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

} // namespace ly
